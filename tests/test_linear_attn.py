"""The mechanisms Femirax is made of, each alone, against their plain equations: decayed linear attention (both decays,
all kernels), rotation + unit norm + cache write, attention over padded and fp32 caches, the fp32 residual update, the
token side input, state slots."""

import pytest
import torch

import femirax_oracle as oracle
from xllm_b200 import ops
from xllm_b200.models.state import RecurrentStatePool
from xllm_b200.ops.linear_attn import LinearAttention
from xllm_b200.ops.residual import gelu_mul_rows, residual_update

TARGETS = [pytest.param(("cpu", torch.float32), id="cpu-fp32"),
           pytest.param(("cuda", torch.float32), id="gpu-fp32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())


def table(rot, base, n=4096):
    a = torch.arange(n, dtype=torch.float64)[:, None] * base ** (-2.0 * torch.arange(rot // 2, dtype=torch.float64) / rot)
    return torch.cat([a.cos(), a.sin()], -1).float()


class Case:
    """Projection rows of some sequences with their plain answers."""

    def __init__(self, target, H, dk, dv, lens, decay=None, rank=0, tau=1.0, bias=3.0, rot=0, interleaved=False, seed=0,
                 gate=True, weight=True):
        self.dev, self.dt = target
        g = torch.Generator().manual_seed(seed)
        T = sum(lens)
        r8 = lambda n: (n + 7) // 8 * 8
        widths = [H * dk, H * dk, H * dv, H * dv] + ([rank] if rank else [])
        at, off = [], 0
        for n in widths:
            at.append((off, n))
            off += r8(n)
        rows = torch.randn(T, off, generator=g).to(self.dt)
        self.rows = rows.to(self.dev)
        self.cols = [self.rows[:, o:o + n] for o, n in at]
        d = [rows[:, o:o + n].double() for o, n in at]
        self.op = LinearAttention(H, dk, dv, q_scale=0.7, k_scale=dk ** -0.5, eps=1e-5)
        if decay is not None:
            self.op.log_decay = torch.log(torch.tensor(decay, dtype=torch.float64)).clamp_min(-700).float().to(self.dev)
        else:
            self.op.a2 = (torch.randn(H * dk, rank, generator=g) * rank ** -0.5).to(self.dt).to(self.dev)
            self.op.a2_bias = (bias + torch.randn(H * dk, generator=g)).to(self.dt).to(self.dev)
            self.op.inv_tau = 1.0 / tau
        if rot:
            self.op.cos_sin, self.op.rot, self.op.interleaved = table(rot, 300.0).to(self.dev), rot, interleaved
        if weight:
            self.op.norm_w = (1 + 0.3 * torch.randn(dv, generator=g)).to(self.dt).to(self.dev)
        self.gate = gate
        self.want, self.bounds, a = [], [], 0
        for n in lens:
            s = slice(a, a + n)
            q, k, v = d[0][s].view(n, H, dk), d[1][s].view(n, H, dk), d[2][s].view(n, H, dv)
            if rot:
                q, k = (oracle.rotate(x, 300.0, rot, "pairs" if interleaved else "half") for x in (q, k))
            if decay is not None:
                al = torch.tensor(decay, dtype=torch.float64).view(1, H, 1).expand(n, H, dk)
            else:
                z = d[4][s] @ self.op.a2.double().cpu().T + self.op.a2_bias.double().cpu()
                al = (1 / (1 + torch.exp(-z))).pow(1 / tau).view(n, H, dk)
            o = oracle.unit_rms(oracle.decayed_state(q * 0.7, k * dk ** -0.5, v, al), 1e-5)
            if weight:
                o = o * self.op.norm_w.double().cpu()
            o = o.reshape(n, H * dv)
            self.want.append(o * oracle.silu(d[3][s]) if gate else o)
            self.bounds.append((a, a + n))
            a += n
        self.state = torch.full((len(lens) + 2, H, dk, (dv + 3) // 4 * 4), 1e9, device=self.dev)   # never read afresh

    def step(self, parts, **kw):
        """parts: (sequence, first, last) token ranges of one prompt batch; returns their rows."""
        idx = torch.cat([torch.arange(self.bounds[s][0] + a, self.bounds[s][0] + b) for s, a, b in parts])
        i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=self.dev)
        rows = self.rows[idx.to(self.dev)]
        cols = [rows[:, c.storage_offset():c.storage_offset() + c.shape[1]] for c in self.cols]
        pos = torch.cat([torch.arange(a, b) for _, a, b in parts]).to(self.dev)
        cu = [0]
        for _, a, b in parts:
            cu.append(cu[-1] + b - a)
        slots, lens = i32([s + 1 for s, _, _ in parts]), i32([b for _, _, b in parts])
        r = cols[4] if len(cols) > 4 else None
        g = cols[3] if self.gate else None
        if kw.pop("decode", False):
            return self.op.decode(self.state, slots, lens, pos, cols[0], cols[1], cols[2], g=g, r=r)
        return self.op.prefill(self.state, slots, i32(cu), lens, pos, cols[0], cols[1], cols[2], g=g, r=r, **kw)

    def check(self, got, parts, tol):
        want = torch.cat([self.want[s][a:b] for s, a, b in parts])
        assert bool(torch.isfinite(got.float()).all())
        assert rel(got, want) < tol, rel(got, want)


SIZES = {"r64": dict(H=3, dk=64, dv=64, decay=[0.98, 0.9995, 0.6], rot=64),
         "r_odd": dict(H=2, dk=26, dv=22, decay=[0.9, 1.0], rot=10, weight=False),
         "r_wide": dict(H=2, dk=128, dv=200, decay=[0.99, 0.999], rot=32, interleaved=True),
         "r_256": dict(H=1, dk=256, dv=96, decay=[0.97], rot=128),
         "r_zero": dict(H=2, dk=32, dv=32, decay=[0.0, 1e-30]),
         "c64": dict(H=2, dk=64, dv=64, rank=16, tau=16.0),
         "c_odd": dict(H=3, dk=18, dv=30, rank=5, tau=2.0, gate=False),
         "c_wide": dict(H=2, dk=128, dv=128, rank=40, tau=8.0, bias=5.0),
         "c_fast": dict(H=2, dk=32, dv=48, rank=8, tau=1.0, bias=-4.0),
         "c_resets": dict(H=2, dk=64, dv=32, rank=8, tau=0.05, bias=0.0)}    # decays of e^-100 beside decays near one


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(SIZES))
def test_linear_attention(name, target):
    tol = 1e-5 if target[1] == torch.float32 else 4e-3
    c = Case(target, lens=(49, 16, 1, 34), **SIZES[name])
    everything = [(0, 0, 49), (1, 0, 16), (2, 0, 1), (3, 0, 34)]
    c.check(c.step(everything), everything, tol)
    # portions of two tokens and more, sequences at unequal progress, the slots still holding the run before
    for cut in (2, 5, 16, 17):
        for s, n in ((0, 49), (3, 34)):
            for a in range(0, n, cut):
                p = [(s, a, min(a + cut, n))]
                c.check(c.step(p), p, tol * 2)
    # the first tokens and the rest decoded; then both kinds of step in turn
    p = [(0, 0, 3), (3, 0, 20)]
    c.check(c.step(p), p, tol)
    for t in range(12):
        p = [(0, 3 + t, 4 + t), (3, 20 + t, 21 + t)]
        c.check(c.step(p, decode=True), p, tol * 3)
    p = [(3, 32, 34), (0, 15, 49)]
    c.check(c.step(p), p, tol * 2)
    p = [(1, 0, 1), (2, 0, 1)]                                  # a first token that is decoded starts from nothing
    c.check(c.step(p, decode=True), p, tol * 2)


@pytest.mark.gpu
@pytest.mark.parametrize("length", [16, 48, 128])
@pytest.mark.parametrize("name", ["r64", "r_odd", "r_wide", "c64", "c_odd", "c_resets"])
def test_segments_side_by_side(name, length, monkeypatch):
    """Long prompts run as segments with a scan over their states; borders of segments, several sequences of unequal
    numbers of segments, continued from a state, and the state they leave."""
    lens = (150, 16, 1, 97)
    c = Case(("cuda", torch.bfloat16), lens=lens, seed=2, **SIZES[name])

    def segments(self, T, n_seqs, max_q_len, device):
        segs = -(-max_q_len // length)
        m = T // length + n_seqs + 1
        nan = float("nan")
        return (torch.full((m, self.heads, self.dk, (self.dv + 3) // 4 * 4), nan, device=device),
                torch.full((m, self.heads, self.dk), nan, device=device), length, segs)

    monkeypatch.setattr(LinearAttention, "_segments", segments)
    p = [(s, 0, n) for s, n in enumerate(lens)]
    c.check(c.step(p, max_q_len=150), p, 4e-3)
    p = [(0, 0, 100), (3, 0, 31)]
    c.check(c.step(p, max_q_len=100), p, 4e-3)
    p = [(3, 31, 96), (0, 100, 149)]
    c.check(c.step(p, max_q_len=65), p, 6e-3)
    p = [(0, 149, 150), (3, 96, 97)]
    c.check(c.step(p, decode=True), p, 8e-3)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["r64", "c64", "c_resets"])
def test_token_by_token_form(name, target):
    c = Case(target, lens=(40, 7), seed=3, **SIZES[name])
    p = [(0, 0, 23), (1, 0, 7)]
    c.check(c.step(p, token_by_token=True), p, 1e-5 if target[1] == torch.float32 else 4e-3)
    p = [(0, 23, 40)]
    c.check(c.step(p), p, 1e-5 if target[1] == torch.float32 else 4e-3)


@pytest.mark.parametrize("target", TARGETS)
def test_padding_rows_touch_no_state(target):
    c = Case(target, lens=(20,), seed=1, **SIZES["c64"])
    p = [(0, 0, 20)]
    c.step(p)
    before = c.state.clone()
    dev = target[0]
    i32 = lambda x: torch.tensor(x, dtype=torch.int32, device=dev)
    cols = [x[:2] for x in c.cols]
    y = c.op.decode(c.state, i32([-1, -1]), i32([0, 0]), torch.zeros(2, dtype=torch.int64, device=dev), cols[0], cols[1],
                    cols[2], g=cols[3], r=cols[4])
    c.op.prefill(c.state, i32([-1, 1]), i32([0, 2, 2]), i32([0, 0]), torch.zeros(20, dtype=torch.int64, device=dev), *c.cols[:3],
                 g=c.cols[3], r=c.cols[4], padded=True)
    assert torch.equal(c.state, before) and float(y.float().abs().max()) == 0.0


# ------------------------------------------------------------------------------------------- rotation, norm, attention
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("nq,nkv,d,rot,interleaved", [(6, 2, 20, 12, True), (4, 4, 64, 64, True), (5, 1, 48, 48, False),
                                                      (3, 3, 128, 32, True), (2, 1, 130, 6, True), (2, 2, 10, 0, False),
                                                      (4, 2, 300, 64, True)])
def test_rotation_unit_norm_and_attention(nq, nkv, d, rot, interleaved, target):
    dev, dt = target
    g = torch.Generator().manual_seed(d)
    lens, page = (37, 16, 5), 16
    T = sum(lens)
    cols = [nq * d, nkv * d]
    rows = torch.randn(T, sum(cols) + 3, generator=g).to(dt)
    rd = rows.double()
    r = rows.to(dev)
    dp = ops.attention_head_size(d)
    kc, vc = (torch.full((12, nkv, page, dp), 7.0, dtype=dt, device=dev) for _ in range(2))
    bt = torch.tensor([[3, 9, 1], [4, 0, 0], [8, 0, 0]], dtype=torch.int32)
    pos, slots = [], []
    for s, n in enumerate(lens):
        for p in range(n):
            pos.append(p)
            slots.append(int(bt[s, p // page]) * page + p % page)
    pos, slots = torch.tensor(pos), torch.tensor(slots, dtype=torch.int32)
    cs = table(rot, 700.0).to(dev) if rot else None
    k_cols = r[:, cols[0]:cols[0] + cols[1]]
    q = ops.rope_norm_kv_write(r[:, :cols[0]], k_cols, k_cols, nq, nkv, d, pos.to(dev), cs, rot, slots.to(dev), kc, vc,
                               eps=1e-5, interleaved=interleaved)
    cu = torch.tensor([0, 37, 53, 58], dtype=torch.int32, device=dev)
    kv = torch.tensor(lens, dtype=torch.int32, device=dev)
    bt = bt.to(dev)
    out = torch.zeros_like(q)
    scale = 2.5 * d ** -0.5
    if dev == "cpu" or dt == torch.float32 or dp not in (64, 128, 256):
        ops.paged_attention_generic(q, kc, vc, bt, cu, kv, scale, out=out)
    else:
        ops.paged_prefill_attention(q, kc, vc, bt, cu, kv, 37, scale, out=out)
        last = cu[1:].long() - 1                                # the last row of each sequence, as a decode row
        dec = ops.paged_decode_attention(q[last].contiguous(), kc, vc, bt, kv, scale)
        assert rel(dec, out[last]) < 1e-2
    gen = ops.paged_attention_generic(q, kc, vc, bt, cu, kv, scale)
    tol = 1e-5 if dt == torch.float32 else 1e-2
    a = 0
    for n in lens:
        s = slice(a, a + n)
        raw = rd[s, cols[0]:cols[0] + cols[1]].view(n, nkv, d)
        qq = rd[s, :cols[0]].view(n, nq, d)
        lay = "pairs" if interleaved else "half"
        if rot:
            qq, kk = oracle.rotate(qq, 700.0, rot, lay), oracle.rotate(raw, 700.0, rot, lay)
        else:
            kk = raw
        want = oracle.causal_attention(oracle.unit_rms(qq, 1e-5), oracle.unit_rms(kk, 1e-5), raw, scale)
        assert rel(out[s, :, :d], want) < tol and rel(gen[s, :, :d], want) < tol
        if dp > d:
            assert float(out[s, :, d:].float().abs().max()) == 0.0
        a += n


# ------------------------------------------------------------------------------------------- residual and side input
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 72, 200, 37, 4096, 5120])
def test_residual_update(H, target):
    dev, dt = target
    g = torch.Generator().manual_seed(H)
    T = 9
    mk = lambda *s: torch.randn(*s, generator=g).to(dt)
    tab, y, y2, w, w2, wo = mk(11, H), mk(T, H), mk(T, H), mk(H), mk(H), mk(H)
    ids = torch.randint(0, 11, (T,), generator=g)
    d = lambda t: t.to(dev)
    tol_x, tol_o = 2e-6, 2e-6 if dt == torch.float32 else 4e-3
    x, out = residual_update(None, d(tab), rows=d(ids), w_out=d(wo), eps=1e-4)
    rx = tab.double()[ids]
    assert rel(x, rx) < tol_x and rel(out, oracle.rms_norm(rx, wo.double(), 1e-4)) < tol_o and x.dtype == torch.float32
    for kw, add in ((dict(), y.double()), (dict(w=d(w)), oracle.rms_norm(y.double(), w.double(), 1e-4)),
                    (dict(w=d(w), y2=d(y2), w2=d(w2), coef=0.5),
                     0.5 * (oracle.rms_norm(y.double(), w.double(), 1e-4) + oracle.rms_norm(y2.double(), w2.double(), 1e-4)))):
        for wout in (None, wo):
            x, out = residual_update(x, d(y), w_out=None if wout is None else d(wout), eps=1e-4, **kw)
            rx = rx + add
            assert rel(x, rx) < tol_x
            assert rel(out, rx if wout is None else oracle.rms_norm(rx, wout.double(), 1e-4)) < tol_o
            assert out.dtype == dt and out.data_ptr() != x.data_ptr()


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("dim", [6, 16, 24])
def test_token_side_activation(dim, target):
    dev, dt = target
    g = torch.Generator().manual_seed(dim)
    width = (dim + 7) // 8 * 8
    gate, tab = (3 * torch.randn(7, width, generator=g)).to(dt), torch.randn(5, 3 * dim, generator=g).to(dt)
    ids = torch.tensor([4, 0, 2, 2, 1, 3, 4])
    got = gelu_mul_rows(gate.to(dev), tab.to(dev), ids.to(dev), 2 * dim, dim)
    want = oracle.gelu_tanh(gate.double()[:, :dim]) * tab.double()[ids][:, 2 * dim:]
    assert rel(got[:, :dim], want) < (2e-6 if dt == torch.float32 else 4e-3)
    assert width == dim or float(got[:, dim:].float().abs().max()) == 0.0


def test_state_pool():
    pool = RecurrentStatePool({1: (2, 8, 6), 3: (1, 4, 4)}, 3, "cpu")
    assert pool.layers[1].shape == (4, 2, 8, 8) and pool.scratch_slot == 3
    assert RecurrentStatePool.bytes_per_slot({1: (2, 8, 6), 3: (1, 4, 4)}) == (2 * 8 * 8 + 16) * 4
    a = [pool.slot_of(i) for i in (10, 11, 12)]
    assert sorted(a) == [0, 1, 2] and pool.slot_of(11) == a[1]
    with pytest.raises(RuntimeError):
        pool.slot_of(13)
    pool.release(11)
    pool.release(11)
    assert pool.slot_of(13) == a[1]
