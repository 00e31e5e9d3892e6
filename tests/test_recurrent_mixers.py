"""The mechanisms Sodedra is made of, each alone, against their plain equations: gated delta rule with channel decays behind
short convolutions, matrix memory with exponential gates, head norms and gates, windowed attention with value heads of
their own size, scaled rotary frequencies, expert routing by groups and grouped expert products, fp32 projections, the
residual update with norm weights stored around zero, states of several parts."""

import pytest
import torch

import sodedra_oracle as oracle
from xllm_b200 import ops
from xllm_b200.models.state import RecurrentStatePool
from xllm_b200.ops import moe as M
from xllm_b200.ops import reference
from xllm_b200.ops.delta_rule import ChannelDelta
from xllm_b200.ops.head_norm import head_gate, head_norm_gate
from xllm_b200.ops.mlstm import MatrixMemory
from xllm_b200.ops.residual import residual_update

TARGETS = [pytest.param(("cpu", torch.float32), id="cpu-fp32"),
           pytest.param(("cuda", torch.float32), id="gpu-fp32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt())


# ------------------------------------------------------------------------------------------- recurrences
class Case:
    """Projection rows of some sequences with their plain answers; slots hold garbage that must never be read afresh."""

    def __init__(self, target, lens):
        self.dev, self.dt = target
        self.bounds, a = [], 0
        for n in lens:
            self.bounds.append((a, a + n))
            a += n
        self.T = a

    def columns(self, g, widths):
        at, off = [], 0
        for n in widths:
            at.append((off, n))
            off += (n + 7) // 8 * 8
        rows = torch.randn(self.T, off, generator=g).to(self.dt)
        self.rows = rows.to(self.dev)
        self.at = at
        return [rows[:, o:o + n].double() for o, n in at]

    def i32(self, x):
        return torch.tensor(x, dtype=torch.int32, device=self.dev)

    def batch(self, parts):
        idx = torch.cat([torch.arange(self.bounds[s][0] + a, self.bounds[s][0] + b) for s, a, b in parts]).to(self.dev)
        rows = self.rows[idx]
        cu = [0]
        for _, a, b in parts:
            cu.append(cu[-1] + b - a)
        return idx, [rows[:, o:o + n] for o, n in self.at], self.i32([s + 1 for s, _, _ in parts]), self.i32(cu), \
            self.i32([b for _, _, b in parts])

    def check(self, got, parts, tol):
        want = torch.cat([self.want[s][a:b] for s, a, b in parts])
        assert bool(torch.isfinite(got.float()).all())
        assert rel(got, want) < tol, rel(got, want)


class DeltaCase(Case):
    def __init__(self, target, H, G, dk, dv, taps, rank, lens, a_log=0.0, bias=-3.0, seed=0):
        super().__init__(target, lens)
        g = torch.Generator().manual_seed(seed)
        mk = lambda *s: torch.randn(*s, generator=g)
        q, k, v, r, gate = self.columns(g, [G * dk, G * dk, H * dv, rank, H * dv])
        self.zb = (2 * mk(self.T, H)).to(self.dev)
        put = lambda t: t.to(self.dt).to(self.dev)
        C = 2 * G * dk + H * dv
        self.op = op = ChannelDelta(H, G, dk, dv, taps, q_scale=dk ** -0.5, eps=1e-5, conv_w=put(mk(C, taps).T.contiguous() * 0.6),
                                    a2=put(mk(H * dk, rank) * rank ** -0.5), dt_bias=put(bias + mk(H * dk)),
                                    a_log=put(a_log + 0.5 * mk(H)), norm_w=put(1 + 0.3 * mk(dv)))
        d = lambda t: t.double().cpu()
        cw, share = d(op.conv_w).T, torch.arange(H) // (H // G)
        unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
        self.want = []
        for a, b in self.bounds:
            n = b - a
            x = oracle.silu(oracle.short_conv(torch.cat([q[a:b], k[a:b], v[a:b]], 1), cw))
            qq, kk, vv = x.split([G * dk, G * dk, H * dv], 1)
            z = oracle.softplus(r[a:b] @ d(op.a2).T + d(op.dt_bias)).view(n, H, dk)
            decay = torch.exp(-torch.exp(d(op.a_log))[None, :, None] * z)
            o = oracle.delta_rule(unit(qq.view(n, G, dk))[:, share] * dk ** -0.5, unit(kk.view(n, G, dk))[:, share],
                                  vv.view(n, H, dv), oracle.sigmoid(d(self.zb)[a:b]), decay)
            o = (oracle.unit_rms(o, 1e-5) * d(op.norm_w)).reshape(n, H * dv)
            self.want.append(o * oracle.sigmoid(gate[a:b]))
        self.state = torch.full((len(lens) + 2, H, dk, (dv + 3) // 4 * 4), 1e9, device=self.dev)
        self.ring = torch.full((len(lens) + 2, taps, C), 1e9, dtype=self.dt, device=self.dev)

    def step(self, parts, decode=False, **kw):
        idx, (q, k, v, r, gate), slots, cu, lens = self.batch(parts)
        out = torch.empty(len(idx), self.op.heads * self.op.dv, dtype=self.dt, device=self.dev)
        run = self.op.decode if decode else self.op.prefill
        return run(self.state, self.ring, slots, cu, lens, q, k, v, r, self.zb[idx], gate, out, **kw)


class MemoryCase(Case):
    def __init__(self, target, H, dk, dv, cap, lens, f_bias=3.0, i_bias=0.0, seed=0):
        super().__init__(target, lens)
        g = torch.Generator().manual_seed(seed)
        mk = lambda *s: torch.randn(*s, generator=g)
        q, k, v, gate = self.columns(g, [H * dk, H * dk, H * dv, H * dv])
        self.z = torch.cat([i_bias + 3 * mk(self.T, H), f_bias + 2 * mk(self.T, H)], 1).to(self.dev)
        self.op = MatrixMemory(H, dk, dv, cap, q_scale=dk ** -0.5, eps=1e-5,
                               norm_w=(1 + 0.3 * mk(H * dv)).to(self.dt).to(self.dev))
        z, w = self.z.double().cpu(), self.op.norm_w.double().cpu()
        self.want = []
        for a, b in self.bounds:
            n = b - a
            i = cap * torch.tanh(z[a:b, :H] / cap)
            f = oracle.log_sigmoid(cap * torch.tanh(z[a:b, H:] / cap))
            o = oracle.stabilised_memory(q[a:b].view(n, H, dk) * dk ** -0.5, k[a:b].view(n, H, dk), v[a:b].view(n, H, dv), i, f)
            self.want.append(oracle.unit_rms(o, 1e-5).reshape(n, H * dv) * w * oracle.sigmoid(gate[a:b]))
        full = lambda *s: torch.full((len(lens) + 2, *s), 1e9, device=self.dev)
        self.state = {"S": full(H, dk, (dv + 3) // 4 * 4), "n": full(H, dk), "m": full(H)}

    def step(self, parts, decode=False, **kw):
        idx, (q, k, v, gate), slots, cu, lens = self.batch(parts)
        H = self.op.heads
        out = torch.empty(len(idx), H * self.op.dv, dtype=self.dt, device=self.dev)
        z = self.z[idx]
        run = self.op.decode if decode else self.op.prefill
        return run(self.state, slots, cu, lens, q, k, v, z[:, :H], z[:, H:], gate, out, **kw)


LENS = (49, 16, 1, 34)
CASES = {
    "delta_64": lambda t, lens=LENS: DeltaCase(t, 2, 2, 64, 64, 4, 16, lens),
    "delta_shared": lambda t, lens=LENS: DeltaCase(t, 6, 2, 32, 48, 3, 8, lens),
    "delta_odd": lambda t, lens=LENS: DeltaCase(t, 3, 1, 18, 30, 2, 5, lens),
    "delta_one_tap": lambda t, lens=LENS: DeltaCase(t, 2, 1, 26, 9, 1, 3, lens),
    "delta_long_conv": lambda t, lens=LENS: DeltaCase(t, 1, 1, 40, 72, 9, 24, lens),
    "delta_128": lambda t, lens=LENS: DeltaCase(t, 2, 2, 128, 128, 4, 128, lens),
    "delta_wide": lambda t, lens=LENS: DeltaCase(t, 2, 1, 200, 160, 4, 40, lens),
    "delta_tall": lambda t, lens=LENS: DeltaCase(t, 1, 1, 300, 40, 4, 8, lens),
    "delta_fast": lambda t, lens=LENS: DeltaCase(t, 2, 2, 64, 32, 4, 8, lens, a_log=2.0, bias=2.0),     # decays of e^-40
    "memory_64": lambda t, lens=LENS: MemoryCase(t, 2, 64, 64, 15.0, lens),
    "memory_odd": lambda t, lens=LENS: MemoryCase(t, 3, 18, 30, 7.0, lens),
    "memory_thin": lambda t, lens=LENS: MemoryCase(t, 4, 32, 9, 4.0, lens),
    "memory_128": lambda t, lens=LENS: MemoryCase(t, 2, 128, 128, 12.0, lens),
    "memory_wide": lambda t, lens=LENS: MemoryCase(t, 1, 200, 160, 20.0, lens),
    "memory_tall": lambda t, lens=LENS: MemoryCase(t, 1, 300, 40, 10.0, lens),
    "memory_strong": lambda t, lens=LENS: MemoryCase(t, 2, 32, 32, 30.0, lens, i_bias=15.0),      # gates of e^25
    "memory_weak": lambda t, lens=LENS: MemoryCase(t, 2, 32, 32, 30.0, lens, i_bias=-12.0),       # the floor e^-m rules
    "memory_forgets": lambda t, lens=LENS: MemoryCase(t, 2, 64, 48, 30.0, lens, f_bias=-12.0),
}


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CASES))
def test_recurrence(name, target):
    tol = 2e-5 if target[1] == torch.float32 else 4e-3
    if name == "memory_forgets":
        tol *= 6        # the output is (k . q) v over its own size: what is left of a k . q that nearly cancels
    c = CASES[name](target)
    everything = [(s, 0, n) for s, n in enumerate(LENS)]
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
    for t in range(1, 8):
        p = [(1, t, t + 1)]
        c.check(c.step(p, decode=True), p, tol * 3)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["delta_64", "memory_64", "delta_128", "memory_128"])
def test_long_prompt(name, target):
    """Many tiles of tokens, several sequences, continued."""
    lens = (330, 17, 205)
    c = CASES[name](target, lens)
    p = [(s, 0, n) for s, n in enumerate(lens)]
    tol = 3e-5 if target[1] == torch.float32 else 5e-3
    c.check(c.step(p), p, tol)
    p = [(2, 0, 100), (0, 0, 65)]
    c.check(c.step(p), p, tol)
    p = [(0, 65, 330), (2, 100, 205)]
    c.check(c.step(p), p, tol)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CASES))
def test_token_by_token_form(name, target):
    """The fp32 recurrence of every type, before and behind the form in chunks."""
    c = CASES[name](target)
    tol = (2e-5 if target[1] == torch.float32 else 4e-3) * (6 if name == "memory_forgets" else 1)
    p = [(0, 0, 23), (1, 0, 16), (3, 0, 2)]
    c.check(c.step(p, token_by_token=True), p, tol)
    p = [(0, 23, 40), (3, 2, 20)]
    c.check(c.step(p), p, tol * 2)
    p = [(0, 40, 49), (3, 20, 34)]
    c.check(c.step(p, token_by_token=True), p, tol * 2)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["delta_64", "memory_64"])
def test_padding_rows_touch_no_state(name, target):
    c = CASES[name](target)
    p = [(0, 0, 20)]
    c.step(p)
    parts = (lambda: [c.state["S"], c.state["n"], c.state["m"]]) if isinstance(c.state, dict) else (lambda: [c.state, c.ring])
    before = [t.clone() for t in parts()]
    idx, cols, slots, cu, lens = c.batch([(0, 0, 20)])
    H, W = c.op.heads, c.op.heads * c.op.dv
    i32, out = c.i32, torch.full((20, W), 7.0, dtype=c.dt, device=c.dev)
    gate = cols[-1]
    if isinstance(c.state, dict):
        args = lambda n: (*[x[:n] for x in cols[:3]], c.z[:n, :H], c.z[:n, H:], gate[:n], out[:n])
        state = (c.state,)
    else:
        args = lambda n: (*[x[:n] for x in cols[:4]], c.zb[:n], gate[:n], out[:n])
        state = (c.state, c.ring)
    if c.dev == "cuda":
        c.op.decode(*state, i32([-1, -1]), i32([0, 1, 2]), i32([0, 0]), *args(2))
        assert float(out[:2].float().abs().max()) == 0.0
        c.op.prefill(*state, i32([-1, 1]), i32([0, 2, 2]), i32([0, 0]), *args(20), padded=True)
        assert float(out.float().abs().max()) == 0.0
    else:
        c.op.prefill(*state, i32([-1, 1]), i32([0, 2, 2]), i32([0, 0]), *args(20), padded=True)
    for a, b in zip(before, parts()):
        assert torch.equal(a, b)


def test_state_of_several_parts():
    shapes = {0: {"S": ((2, 8, 6), None), "conv": ((3, 10), torch.bfloat16)}, 2: (1, 4, 4), 3: {"n": ((2, 5), torch.float32)}}
    pool = RecurrentStatePool(shapes, 3, "cpu")
    assert pool.layers[0]["S"].shape == (4, 2, 8, 8) and pool.layers[0]["S"].dtype == torch.float32
    assert pool.layers[0]["conv"].shape == (4, 3, 10) and pool.layers[0]["conv"].dtype == torch.bfloat16
    assert pool.layers[2].shape == (4, 1, 4, 4) and pool.layers[3]["n"].shape == (4, 2, 5)
    assert RecurrentStatePool.bytes_per_slot(shapes) == 2 * 8 * 8 * 4 + 30 * 2 + 16 * 4 + 10 * 4


# ------------------------------------------------------------------------------------------- head norms and gates
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H,dv", [(3, 30), (2, 64), (4, 9), (1, 200), (2, 600), (5, 128)])
def test_head_norm_and_gate(H, dv, target):
    dev, dt = target
    g = torch.Generator().manual_seed(dv)
    T = 7
    o, div = torch.randn(T, H, dv, generator=g), torch.rand(T, H, generator=g) + 0.1
    gate = torch.randn(T, H * dv + 8, generator=g).to(dt)[:, :H * dv]
    tol = 2e-6 if dt == torch.float32 else 4e-3
    for n_w in (0, dv, H * dv):
        w = (1 + torch.randn(n_w, generator=g)).to(dt) if n_w else None
        for act in ("silu", "sigmoid"):
            for use_div in (False, True):
                out = torch.empty(T, H * dv, dtype=dt, device=dev)
                head_norm_gate(o.to(dev), out, div=div.to(dev) if use_div else None, g=gate.to(dev),
                               w=w.to(dev) if n_w else None, act=act, eps=1e-3)
                x = o.double() / (div.double()[..., None] if use_div else 1.0)
                x = oracle.unit_rms(x, 1e-3)
                if n_w:
                    x = x * w.double().view(-1, dv)
                z = gate.double()
                want = x.reshape(T, H * dv) * (oracle.silu(z) if act == "silu" else oracle.sigmoid(z))
                assert rel(out, want) < tol
    a = torch.randn(T, H, dv + 8, generator=g).to(dt)
    assert rel(head_gate(a.to(dev), gate.to(dev), dv), a.double()[..., :dv].reshape(T, -1) * oracle.sigmoid(gate.double())) < tol


# ------------------------------------------------------------------------------------------- attention
@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 64), (8.0, 2.0, 2.0, 100), (1.0, 1.0, 3.0, 50)])
def test_rotary_frequencies(scaling):
    """Kept below, divided beyond, a ramp in between."""
    names = dict(zip(("factor", "low", "high", "original"), scaling)) if scaling else None
    s = {"rope_type": "llama3", "factor": scaling[0], "low_freq_factor": scaling[1], "high_freq_factor": scaling[2],
         "original_max_position_embeddings": scaling[3]} if scaling else None
    table = reference.build_cos_sin_cache(24, 300, 900.0, s)
    x = torch.zeros(300, 1, 24, dtype=torch.float64)
    x[:, :, :12] = 1.0
    y = oracle.rotate(x, 900.0, 24, names)
    assert float((table[:, :12] - y[:, 0, :12]).abs().max()) < 1e-6 and float((table[:, 12:] - y[:, 0, 12:]).abs().max()) < 1e-6


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("nq,nkv,d,dv,rot,window", [(6, 2, 20, 12, 12, 1), (4, 2, 24, 40, 24, 2), (4, 4, 64, 64, 16, 16),
                                                    (4, 1, 128, 128, 64, 37), (4, 2, 128, 96, 128, 128), (2, 1, 128, 128, 16, 129),
                                                    (3, 1, 128, 128, 32, 200), (2, 2, 70, 130, 10, 64), (3, 3, 300, 20, 8, 33),
                                                    (2, 1, 64, 64, 64, 1000)])
def test_windowed_attention(nq, nkv, d, dv, rot, window, target):
    """Rotation of the first elements, cache write with value heads of their own size, window: whole prompts and their last
    rows as decode rows.  Pages wholly before a window are given back (their table entries name block 0)."""
    dev, dt = target
    g = torch.Generator().manual_seed(d + window)
    lens, page = (300, 16, 141), 16
    cols = [nq * d, nkv * d, nkv * dv]
    rows = torch.randn(sum(lens), sum(cols) + 8, generator=g).to(dt)
    r, rd = rows.to(dev), rows.double()
    dp = ops.attention_head_size(max(d, dv))
    n_pages = [(n + page - 1) // page for n in lens]
    order = (torch.randperm(sum(n_pages), generator=g) + 1).tolist()
    bt = torch.zeros(3, max(n_pages), dtype=torch.int32)
    pos, slots = [], []
    for s, n in enumerate(lens):
        for i in range(n_pages[s]):
            bt[s, i] = order.pop()
        for p in range(n):
            pos.append(p)
            slots.append(int(bt[s, p // page]) * page + p % page)
    kc, vc = (torch.zeros(sum(n_pages) + 1, nkv, page, dp, dtype=dt, device=dev) for _ in range(2))
    cs = reference.build_cos_sin_cache(rot, 400, 700.0, None, dev)
    q = ops.rope_norm_kv_write(r[:, :cols[0]], r[:, cols[0]:cols[0] + cols[1]], r[:, cols[0] + cols[1]:sum(cols)], nq, nkv, d,
                               torch.tensor(pos, device=dev), cs, rot, torch.tensor(slots, dtype=torch.int32, device=dev), kc, vc,
                               unit_norm=False)
    cu = torch.tensor([0, 300, 316, 457], dtype=torch.int32, device=dev)
    kv = torch.tensor(lens, dtype=torch.int32, device=dev)
    scale = 1.5 * d ** -0.5
    dead = bt.clone()
    for s, n in enumerate(lens):
        dead[s, :max(0, n - window) // page] = 0
    bt, dead = bt.to(dev), dead.to(dev)
    outs = [ops.paged_attention_generic(q, kc, vc, bt, cu, kv, scale, window=window)]
    last = cu[1:].long() - 1
    decs = []
    if dev == "cuda" and dt == torch.bfloat16 and dp in (64, 128, 256):
        outs.append(ops.paged_prefill_attention(q, kc, vc, bt, cu, kv, 300, scale, window=window, out=torch.zeros_like(q)))
        decs = [ops.paged_decode_attention(q[last].contiguous(), kc, vc, dead, kv, scale, window=window, splits=n) for n in (1, 3)]
        # the last 130 tokens of the first sequence as a portion, what lies before its window given back
        gone = bt[:1].clone()
        gone[0, :max(0, 170 - window + 1) // page] = 0
        part = ops.paged_prefill_attention(q, kc, vc, gone, torch.tensor([170, 300], dtype=torch.int32, device=dev), kv[:1], 130,
                                           scale, window=window, out=torch.zeros_like(q))
        assert rel(part[170:300], outs[1][170:300]) < 1e-2
    elif dev == "cpu":
        decs = [ops.paged_decode_attention(q[last], kc, vc, dead, kv, scale, window=window)]
    tol = 1e-5 if dt == torch.float32 else 1e-2
    a = 0
    for s, n in enumerate(lens):
        at = slice(a, a + n)
        x = rd[at]
        qq = oracle.rotate(x[:, :cols[0]].reshape(n, nq, d), 700.0, rot)
        kk = oracle.rotate(x[:, cols[0]:cols[0] + cols[1]].reshape(n, nkv, d), 700.0, rot)
        want = oracle.window_attention(qq, kk, x[:, cols[0] + cols[1]:sum(cols)].reshape(n, nkv, dv), scale, window)
        for out in outs:
            assert rel(out[at][..., :dv], want) < tol
            assert dp == dv or float(out[at][..., dv:].float().abs().max()) == 0.0
        for dec in decs:
            assert rel(dec[s, :, :dv], want[-1]) < tol * 2
        a += n


# ------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("E,groups,keep,K", [(12, 3, 2, 4), (10, 5, 5, 3), (6, 1, 1, 6), (64, 8, 3, 8), (9, 9, 4, 4), (8, 2, 1, 1)])
def test_routing_by_groups(E, groups, keep, K, target):
    """Groups rank by their best corrected score, corrections push scores below zero, weights come from plain scores."""
    dev, _ = target
    g = torch.Generator().manual_seed(E)
    T = 40
    z, c = 2 * torch.randn(T, E + 8, generator=g)[:, :E], 0.6 * torch.randn(E, generator=g) - 0.4
    ids, w = oracle.route(z.double(), c.double(), K, groups, keep, 1.7)
    want = torch.zeros(T, E, dtype=torch.float64).scatter_(1, ids, w)
    if dev == "cpu":
        gi, gw = M.route_reference(z, K, "softmax", c, groups, keep, True, 1.7, group_score="max")
    else:
        from xllm_b200.ops import _lib
        from xllm_b200.ops._lib import ptr, stream
        ws = M.MoeWorkspace(T, K, E, E, 64, 64, dev)
        zd, cd = torch.randn(T, E + 8, device=dev), c.to(dev)
        zd[:, :E] = z.to(dev)
        assert _lib.load().xllm_moe_route_ld(ptr(zd), E + 8, 1, ptr(cd), ptr(ws.topk_ids), ptr(ws.topk_w), ptr(ws.counts),
                                             ptr(ws.slot), T, E, K, groups, keep, 2, 1, 1.7, 0, E, stream()) == 0
        gi, gw = ws.topk_ids.view(-1)[:T * K].view(T, K).long(), ws.topk_w[:T * K].view(T, K)
    got = torch.zeros(T, E, dtype=torch.float64).scatter_(1, gi.cpu(), gw.double().cpu())
    assert float((got - want).abs().max()) < 1e-5


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("W,ff,E,K,groups,keep,T", [(72, 20, 6, 2, 3, 2, 33), (128, 64, 8, 3, 4, 2, 70), (100, 12, 5, 5, 1, 1, 9),
                                                    (320, 192, 12, 1, 2, 1, 1), (64, 128, 4, 2, 1, 1, 300)])
def test_expert_layer(W, ff, E, K, groups, keep, T, target):
    """A whole expert layer as the model builds it (padded widths, loaders), against one expert at a time."""
    dev, dt = target
    from sodedra_common import config, mlstm, moe
    from xllm_b200.models import create_model, model_args_from_dict
    g = torch.Generator().manual_seed(W)
    cfg = config([mlstm(1, 8, 8, mlp=moe(E, K, ff, 1.3, (groups, keep)))], vocab=16, width=W)
    w = oracle.random_weights(cfg, (4, 4), 3)
    model = create_model(model_args_from_dict(cfg), dt, dev)
    model.load_weights(w.items())
    layer = model.layers[0]
    h = torch.randn(T, W, generator=g).to(dt)
    z = layer.small(h.to(dev))
    y = layer.mlp(h.to(dev), logits=layer.small.part(z, "mlp.router"))
    want = oracle.experts(h.double(), {n[len("l0.mlp."):]: t.double() for n, t in w.items() if ".mlp." in n}, cfg["layers"][0]["mlp"])
    assert y.shape == (T, W) and rel(y, want) < (1e-5 if dt == torch.float32 else 1e-2)


# ------------------------------------------------------------------------------------------- projections, residual
@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("T,N,K", [(1, 1, 64), (5, 12, 72), (33, 40, 320), (17, 100, 4096), (1500, 33, 520), (4, 7, 30)])
def test_fp32_projection(T, N, K, target):
    dev, dt = target
    g = torch.Generator().manual_seed(N)
    x, w, b = torch.randn(T, K, generator=g).to(dt), torch.randn(N, K, generator=g).to(dt), torch.randn(N, generator=g).to(dt)
    for bias in (None, b):
        y = ops.linear_f32(x.to(dev), w.to(dev), None if bias is None else bias.to(dev))
        want = x.double() @ w.double().T + (0 if bias is None else b.double())
        assert y.dtype == torch.float32 and y.shape == (T, N) and rel(y, want) < 2e-6


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("H", [64, 37, 4096])
def test_residual_with_centred_norms(H, target):
    dev, dt = target
    g = torch.Generator().manual_seed(H)
    mk = lambda *s: torch.randn(*s, generator=g).to(dt)
    tab, y, y2, wo = mk(11, H), mk(9, H), mk(9, H), mk(H) * 0.2
    ids = torch.randint(0, 11, (9,), generator=g)
    d = lambda t: t.to(dev)
    x, out = residual_update(None, d(tab), rows=d(ids), coef=3.5, w_out=d(wo), eps=1e-4, w_out_offset=1.0)
    rx = tab.double()[ids] * 3.5
    tol = 2e-6 if dt == torch.float32 else 4e-3
    assert rel(x, rx) < 2e-6 and rel(out, oracle.centred_norm(rx, wo.double(), 1e-4)) < tol
    for second in (None, y2):
        x, out = residual_update(x, d(y), y2=None if second is None else d(second), w_out=d(wo), eps=1e-4, w_out_offset=1.0)
        rx = rx + y.double() + (0 if second is None else second.double())
        assert rel(x, rx) < 2e-6 and rel(out, oracle.centred_norm(rx, wo.double(), 1e-4)) < tol
