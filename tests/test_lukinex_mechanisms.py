"""The mechanisms of Lukinex alone against plain implementations: windowed attention with kept first tokens and soft caps on
every kernel, convolution + norm + rotation + cache write, lightning attention, norms of whole rows, latent attention in both
forms, clamped activations, routing, residual updates with a normed sum."""
import math

import pytest
import torch

import lukinex_oracle as oracle
from xllm_b200 import ops
from xllm_b200.ops import glu, mla
from xllm_b200.ops import moe as moe_ops
from xllm_b200.ops.head_norm import head_norm_gate
from xllm_b200.ops.linear_attn import LinearAttention
from xllm_b200.ops.residual import residual_update

KINDS = [pytest.param(("cpu", torch.float32), id="cpu-fp32"),
         pytest.param(("cuda", torch.float32), id="gpu-fp32", marks=pytest.mark.gpu),
         pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def gen(seed):
    return torch.Generator().manual_seed(seed)


def randn(*shape, seed=0, kind=("cpu", torch.float32), scale=1.0):
    """The values as the kernels get them and as float64."""
    t = (torch.randn(*shape, generator=gen(seed)) * scale).to(kind[1])
    return t.to(kind[0]), t.double()


def near(got, want, kind, tight=2e-5, loose=0.012):
    d = (got.double().cpu() - want).abs().max() / want.abs().max().clamp_min(1e-6)
    assert float(d) < (loose if kind[1] == torch.bfloat16 else tight), float(d)


def i32(x, kind):
    return torch.tensor(x, dtype=torch.int32, device=kind[0])


class Paged:
    """Sequences of given lengths in a shuffled page pool; `new` of each one's tokens are this step's rows (decode rows first)."""

    def __init__(self, lens, new, kind, page=16, seed=0):
        n_pages = [-(-l // page) for l in lens]
        order = (torch.randperm(sum(n_pages), generator=gen(seed)) + 1).tolist()
        width = max(n_pages)
        self.table, at = [], 0
        for n in n_pages:
            self.table.append(order[at:at + n] + [0] * (width - n))
            at += n
        self.blocks, self.page, self.lens, self.new, self.kind = sum(n_pages) + 1, page, lens, new, kind
        self.n_decode = sum(1 for n in new if n == 1)
        assert all(n == 1 for n in new[:self.n_decode])
        cu = [0]
        for n in new:
            cu.append(cu[-1] + n)
        self.cu = cu
        self.block_table, self.kv_lens, self.cu_q = i32(self.table, kind), i32(lens, kind), i32(cu, kind)
        pos = [p for l, n in zip(lens, new) for p in range(l - n, l)]
        self.positions = torch.tensor(pos, device=kind[0])
        self.slots = i32([self.slot(s, p) for s, (l, n) in enumerate(zip(lens, new)) for p in range(l - n, l)], kind)

    def slot(self, s, p):
        return self.table[s][p // self.page] * self.page + p % self.page

    def cache(self, heads, d, fill=float("nan")):
        return torch.full((self.blocks, heads, self.page, d), fill, dtype=self.kind[1], device=self.kind[0])

    def put(self, cache, s, rows):
        """rows [tokens, heads, d] of sequence s into its pages."""
        for p in range(rows.shape[0]):
            sl = self.slot(s, p)
            cache[sl // self.page, :, sl % self.page, :rows.shape[-1]] = rows[p].to(cache)


# ------------------------------------------------------------------------------------------- attention
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("d,heads,kv", [(64, 6, 2), (128, 4, 1), (256, 2, 2), (72, 3, 3)])
@pytest.mark.parametrize("window,keep,cap", [(0, 0, 0.0), (0, 0, 3.0), (20, 5, 0.0), (64, 64, 0.0), (37, 150, 2.0), (130, 16, 6.0),
                                             (1, 1, 0.0), (17, 0, 4.0)])
def test_kept_windows_and_soft_caps(d, heads, kv, window, keep, cap, kind):
    """Decoding and prompt portions over shuffled pages; pages that nobody may read hold NaN."""
    lens, new = [190, 33, 300, 161, 90], [1, 1, 300, 60, 2]
    b = Paged(lens, new, kind)
    kc, vc = b.cache(kv, d), b.cache(kv, d)
    q, q64 = randn(b.cu[-1], heads, d, seed=1, kind=kind, scale=1.5)
    want = torch.zeros(b.cu[-1], heads, d, dtype=torch.float64)
    for s, (l, n) in enumerate(zip(lens, new)):
        k, k64 = randn(l, kv, d, seed=10 + s, kind=kind)
        v, v64 = randn(l, kv, d, seed=20 + s, kind=kind)
        b.put(kc, s, k)
        b.put(vc, s, v)
        full = torch.zeros(l, heads, d, dtype=torch.float64)
        full[l - n:] = q64[b.cu[s]:b.cu[s + 1]]
        mask = oracle.visible(l, window or None, keep if window else 0)
        want[b.cu[s]:b.cu[s + 1]] = oracle.attention(full, k64, v64, d ** -0.5, mask, cap or None)[l - n:]
        # what lies between the kept tokens and the first query's window was given back
        lo, hi = -(-keep // 16), max(0, l - n - window + 1) // 16
        if window:
            for p in range(lo, hi):
                kc[b.table[s][p]] = vc[b.table[s][p]] = float("nan")
                b.block_table[s, p] = 0
    for c in (kc, vc):                                                # rows behind a sequence's end are never anything but zeros
        for s, l in enumerate(lens):
            if l % 16:
                c[b.table[s][l // 16], :, l % 16:] = 0.0
        c[0] = 0.0
    seen = dict(window=window, keep=keep, softcap=cap)
    nd, out = b.n_decode, torch.zeros_like(q)
    if q.is_cuda and (kind[1] != torch.bfloat16 or d == 72):
        ops.paged_attention_generic(q, kc, vc, b.block_table, b.cu_q, b.kv_lens, d ** -0.5, out=out, **seen)
    else:
        for splits in (1, 3):
            ops.paged_decode_attention(q[:nd], kc, vc, b.block_table[:nd], b.kv_lens[:nd], d ** -0.5, out=out[:nd],
                                       splits=splits, **seen)
            near(out[:nd], want[:nd], kind)
        ops.paged_prefill_attention(q, kc, vc, b.block_table[nd:], b.cu_q[nd:], b.kv_lens[nd:], max(new), d ** -0.5, out=out, **seen)
    near(out, want, kind)


def test_soft_cap_bounds_scores():
    s = torch.tensor([-1e4, -30.0, -1e-3, 0.0, 1e-3, 2.0, 1e4])
    k = torch.zeros(1, 1, 16, 16)
    k[0, 0, :7, 0] = s
    q = torch.zeros(1, 1, 16)
    q[0, 0, 0] = 1.0
    v = torch.eye(16)[None, None]
    out = ops.paged_decode_attention(q, k, v, i32([[0]], ("cpu",)), i32([7], ("cpu",)), 1.0, softcap=5.0)
    assert torch.allclose(out[0, 0, :7], torch.softmax(5.0 * torch.tanh(s / 5.0), 0), atol=1e-6)


# ------------------------------------------------------------------------------------------- projections to attention
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("taps", [0, 1, 2, 3, 4, 7])
@pytest.mark.parametrize("heads,kv,d,dv,rot,norm", [(4, 2, 64, 64, 64, False), (6, 1, 128, 128, 64, True), (3, 3, 32, 80, 32, True),
                                                    (4, 2, 64, 24, 0, False), (3, 1, 26, 14, 12, True), (2, 2, 200, 136, 40, False)])
def test_convolution_norm_rotation_and_cache_write(heads, kv, d, dv, rot, norm, taps, kind):
    """Three sequences fed in portions of unequal sizes beside one another, some one token at a time, with other slots and
    padding rows in the batch."""
    dev, dt = kind
    dp = ops.attention_head_size(max(d, dv))
    C = heads * d + kv * (d + dv)
    total = [41, 9, 26]
    xs = [randn(n, C, seed=s, kind=kind) for s, n in enumerate(total)]
    cw, cw64 = randn(taps or 1, C, seed=7, kind=kind, scale=0.5)
    qw, qw64 = randn(d, seed=8, kind=kind)
    kw, kw64 = randn(d, seed=9, kind=kind)
    spec = {"dims": rot, "base": 300.0, "scaling": {"factor": 1.5}}
    cs = ops.reference.build_cos_sin_cache(rot, 64, 300.0, {"rope_type": "linear", "factor": 1.5}, dev) if rot else None
    want = []
    for n, (_, x) in zip(total, xs):
        y = oracle.short_conv(x, cw64.T) if taps else x
        q, k, v = y.split([heads * d, kv * d, kv * dv], dim=1)
        q, k = q.reshape(n, heads, d), k.reshape(n, kv, d)
        if norm:
            q, k = oracle.rms_norm(q, qw64, 1e-5), oracle.rms_norm(k, kw64, 1e-5)
        if rot:
            q, k = oracle.rotate(q, spec), oracle.rotate(k, spec)
        want.append((q, k, v.reshape(n, kv, dv)))
    ring = torch.full((5, max(taps, 1), C), float("nan"), dtype=dt, device=dev)
    slot_of = [3, 0, 2]
    kc, vc = (torch.zeros(12, kv, 16, dp, dtype=dt, device=dev) for _ in range(2))
    pages = [[1, 5, 9], [4, 0, 0], [7, 2, 0]]
    at = [0, 0, 0]
    got_q = [[], [], []]
    for sizes in ([1, 5, 0], [2, 1, 3], [1, 1, 1], [13, 0, 7], [1, 2, 2], [23, 0, 13]):
        live = sorted((s for s in range(3) if sizes[s]), key=lambda s: sizes[s] > 1)
        rows, pos, slots, cu = [], [], [], [0]
        for s in live:
            rows.append(xs[s][0][at[s]:at[s] + sizes[s]])
            for p in range(at[s], at[s] + sizes[s]):
                pos.append(p)
                slots.append(pages[s][p // 16] * 16 + p % 16)
            cu.append(cu[-1] + sizes[s])
        pad = 2                                                       # rows of no sequence
        x = torch.cat(rows + [torch.zeros(pad, C, dtype=dt, device=dev)])
        wide = torch.zeros(x.shape[0], C + 8, dtype=dt, device=dev)   # column blocks of wider rows
        wide[:, :C] = x
        q, k, v = wide[:, :heads * d], wide[:, heads * d:(heads + kv) * d], wide[:, (heads + kv) * d:C]
        conv = None
        if taps:
            conv = (cw, ring, i32([slot_of[s] for s in live], kind), i32(cu, kind), i32([at[s] + sizes[s] for s in live], kind))
        out = ops.rope_norm_kv_write(q, k, v, heads, kv, d, torch.tensor(pos + [0] * pad, device=dev), cs, rot,
                                     i32(slots + [-1] * pad, kind), kc, vc, eps=1e-5, unit_norm=False, q_w=qw if norm else None,
                                     k_w=kw if norm else None, conv=conv, long_portions=max(sizes) > 1)
        assert bool(torch.isfinite(out).all()) and not bool(out[..., d:].any())
        for j, s in enumerate(live):
            got_q[s].append(out[cu[j]:cu[j + 1], :, :d])
            at[s] += sizes[s]
    assert at == total
    for s in range(3):
        q, k, v = want[s]
        near(torch.cat(got_q[s]), q, kind)
        idx = [pages[s][p // 16] * 16 + p % 16 for p in range(total[s])]
        flat = lambda c: c.permute(0, 2, 1, 3).reshape(-1, kv, dp)[idx]
        near(flat(kc)[..., :d], k, kind)
        near(flat(vc)[..., :dv], v, kind)
        assert not bool(flat(kc)[..., d:].any()) and not bool(flat(vc)[..., dv:].any())


# ------------------------------------------------------------------------------------------- lightning attention
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,dk,dv", [(3, 32, 32), (2, 128, 128), (2, 64, 100), (5, 18, 34), (1, 200, 160), (12, 64, 64)])
def test_lightning_attention(heads, dk, dv, kind):
    """Silu on q, k and v, constant decays from strong to none, all heads normed together: whole, in portions, by token."""
    dev, dt = kind
    T, decay = 150, torch.linspace(0.3, 1.0, heads).tolist() if heads > 1 else [0.999]
    op = LinearAttention(heads, dk, dv, eps=1e-5, in_silu=True, rows=True)
    op.log_decay = torch.log(torch.tensor(decay, dtype=torch.float64)).float().to(dev)
    nw, nw64 = randn(heads * dv, seed=4, kind=kind)
    op.norm_w = nw
    ld = heads * (2 * dk + 2 * dv)
    x, x64 = randn(2 * T, ld, seed=3, kind=kind, scale=0.7)
    cut = lambda r: r.split([heads * dk, heads * dk, heads * dv, heads * dv], dim=1)
    want = []
    for s in range(2):
        q, k, v, g = cut(x64[s * T:(s + 1) * T])
        o = oracle.lightning(oracle.silu(q).view(T, heads, dk), oracle.silu(k).view(T, heads, dk), oracle.silu(v).view(T, heads, dv), decay)
        want.append(oracle.rms_norm(o.reshape(T, heads * dv), nw64, 1e-5) * oracle.sigmoid(g))
    state = torch.full((4, heads, dk, (dv + 3) // 4 * 4), float("nan"), device=dev)
    for cuts in ([T], [70, 2, 78], [64, 1, 1, 15, 69]):
        got, at = [[], []], 0
        for n in cuts:
            rows = torch.cat([x[s * T + at:s * T + at + n] for s in range(2)])
            q, k, v, g = cut(rows)
            slots, lens = i32([2, 1], kind), i32([at + n, at + n], kind)
            pos = torch.arange(at, at + n, device=dev).repeat(2)
            if n == 1:
                o = op.decode(state, slots, lens, pos, q, k, v, g=g, out=torch.empty(2, heads * dv, dtype=dt, device=dev))
            else:
                o = op.prefill(state, slots, i32([0, n, 2 * n], kind), lens, pos, q, k, v, g=g)
            for s in range(2):
                got[s].append(o[s * n:(s + 1) * n])
            at += n
        for s in range(2):
            near(torch.cat(got[s]), want[s], kind, loose=0.02)


@pytest.mark.parametrize("kind", KINDS)
def test_slow_decays_stay_exact(kind):
    """A state summed over thousands of tokens under a decay next to one, token by token."""
    dev, dt = kind
    op = LinearAttention(1, 8, 8)
    decay = 0.99973
    op.log_decay = torch.log(torch.tensor([decay], dtype=torch.float64)).float().to(dev)
    op.unit_norm = False
    T = 6000
    q = torch.zeros(T, 8, dtype=dt, device=dev)
    k, v = torch.zeros_like(q), torch.zeros_like(q)
    k[:, 0] = v[:, 0] = 1.0
    q[-1, 0] = 1.0
    state = torch.zeros(1, 1, 8, 8, device=dev)
    pos = torch.arange(T, device=dev)
    op.prefill(state, i32([0], kind), i32([0, T - 1], kind), i32([T - 1], kind), pos, q[:-1], k[:-1], v[:-1])
    op.decode(state, i32([0], kind), i32([T], kind), pos[-1:], q[-1:], k[-1:], v[-1:])
    want = (1 - decay ** T) / (1 - decay)
    assert abs(float(state[0, 0, 0, 0]) / want - 1) < (2e-6 if dt == torch.float32 else 2e-4)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("H,dv", [(1, 96), (1, 513), (1, 4096), (1, 6000), (3, 700), (1, 10)])
def test_norm_and_gate_of_rows(H, dv, kind):
    o, o64 = randn(9, H, dv, seed=1)
    o = o.to(kind[0])
    g, g64 = randn(9, H * dv, seed=2, kind=kind)
    w, w64 = randn(H * dv, seed=3, kind=kind)
    out = torch.empty(9, H * dv, dtype=kind[1], device=kind[0])
    head_norm_gate(o, out, g=g, w=w, act="sigmoid", eps=1e-5)
    want = oracle.rms_norm(o64, w64.view(H, dv), 1e-5).reshape(9, -1) * oracle.sigmoid(g64)
    near(out, want, kind)


# ------------------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("q_rank,rank", [(40, 24), (64, 128), (33, 50), (1536, 512), (4200, 300)])
def test_latent_norms_and_cache_rows(q_rank, rank, kind):
    dev, dt = kind
    T, ld = 7, (q_rank + 7) // 8 * 8 + (rank + 7) // 8 * 8
    rows, r64 = randn(T, ld, seed=1, kind=kind)
    c0 = (q_rank + 7) // 8 * 8
    qw, qw64 = randn(q_rank, seed=2, kind=kind)
    cw, cw64 = randn(rank, seed=3, kind=kind)
    width = mla.latent_width(rank, dt, dev)
    cache = torch.full((4, 1, 16, width), 7.0, dtype=dt, device=dev)
    slots = [17, 16, -1, 40, 63, 18, 5]
    q = mla.latent_norm(rows[:, :q_rank], qw, c0, 1e-5, c=rows[:, c0:c0 + rank], c_w=cw, slots=i32(slots, kind), cache=cache)
    near(q[:, :q_rank], oracle.rms_norm(r64[:, :q_rank], qw64, 1e-5), kind)
    assert not bool(q[:, q_rank:].any())
    flat, want = cache.view(-1, width), oracle.rms_norm(r64[:, c0:c0 + rank], cw64, 1e-5)
    for t, s in enumerate(slots):
        if s >= 0:
            near(flat[s, :rank], want[t], kind)
            assert not bool(flat[s, rank:].any())
    untouched = [s for s in range(64) if s not in slots]
    assert bool((flat[untouched] == 7.0).all())
    near(mla.latent_norm(rows[:, :q_rank], qw, c0, 1e-5)[:, :q_rank], oracle.rms_norm(r64[:, :q_rank], qw64, 1e-5), kind)   # alone


@pytest.mark.gpu
@pytest.mark.parametrize("heads", [1, 7, 16, 20, 33])
@pytest.mark.parametrize("width", mla.LATENT_WIDTHS)
def test_latent_decode_kernel(width, heads):
    """One row per sequence and rows of prompt portions, any split of the context."""
    kind = ("cuda", torch.bfloat16)
    lens, new = [1, 16, 17, 250, 700, 90], [1, 1, 1, 1, 1, 30]
    b = Paged(lens, new, kind)
    cache = b.cache(1, width, fill=0.0)
    c64 = []
    for s, l in enumerate(lens):
        c, c6 = randn(l, 1, width, seed=s, kind=kind)
        b.put(cache, s, c)
        c64.append(c6)
    q, q64 = randn(b.cu[-1], heads, width, seed=50, kind=kind, scale=1.5)
    want = torch.zeros(b.cu[-1], heads, width, dtype=torch.float64)
    for s, (l, n) in enumerate(zip(lens, new)):
        full = torch.zeros(l, heads, width, dtype=torch.float64)
        full[l - n:] = q64[b.cu[s]:b.cu[s + 1]]
        want[b.cu[s]:b.cu[s + 1]] = oracle.attention(full, c64[s], c64[s], width ** -0.5, oracle.visible(l))[l - n:]
    nd = b.n_decode
    for splits in (None, 1, 2, 5):
        got = mla.latent_decode(q[:nd], cache, b.block_table, width ** -0.5, seq_lens=b.kv_lens[:nd], splits=splits)
        near(got, want[:nd], kind)
        got = mla.latent_decode(q[nd:], cache, b.block_table, width ** -0.5, positions=b.positions[nd:],
                                bt_rows=torch.full((30,), 5, dtype=torch.int32, device="cuda"), splits=splits)
        near(got, want[nd:], kind)


@pytest.mark.gpu
def test_gathered_latents_and_attention_over_rows():
    """Dense rows of a few sequences' latents, zeros behind each, and prompt attention whose keys and values are rows."""
    kind = ("cuda", torch.bfloat16)
    lens, new, heads = [200, 33, 129], [150, 33, 2], 3
    b = Paged(lens, new, kind, seed=3)
    cache = b.cache(1, 128, fill=float("nan"))
    for s, l in enumerate(lens):
        b.put(cache, s, randn(l, 1, 128, seed=s, kind=kind)[0])
    per = 208
    rows = mla.latent_gather(cache, b.block_table, b.kv_lens, per)
    for s, l in enumerate(lens):
        assert torch.equal(rows[s * per:s * per + l], randn(l, 1, 128, seed=s, kind=kind)[0][:, 0])
        assert not bool(rows[s * per + l:(s + 1) * per].any())
    kv, kv64 = randn(3 * per, 2 * heads * 128, seed=9, kind=kind)
    q, q64 = randn(b.cu[-1], heads, 128, seed=10, kind=kind)
    out = torch.zeros_like(q)
    pages = torch.arange(3 * per // 16, dtype=torch.int32, device="cuda").view(3, -1)
    ops.ragged_prefill_attention(q, kv[:, :heads * 128], kv[:, heads * 128:], pages, 16, b.cu_q, b.kv_lens, 150, 0.1, out)
    for s, (l, n) in enumerate(zip(lens, new)):
        k, v = (x[s * per:s * per + l].reshape(l, heads, 128) for x in kv64.split(heads * 128, dim=1))
        full = torch.zeros(l, heads, 128, dtype=torch.float64)
        full[l - n:] = q64[b.cu[s]:b.cu[s + 1]]
        near(out[b.cu[s]:b.cu[s + 1]], oracle.attention(full, k, v, 0.1, oracle.visible(l))[l - n:], kind)


# ------------------------------------------------------------------------------------------- feed-forward
def test_clamped_activation_values():
    gate = torch.tensor([-50.0, -2.0, 0.0, 0.3, 1.5, 1.6, 90.0]).double()
    for limit in (0.5, 1.5, 7.0):
        for up in (-9.0, -limit, -0.2, 0.0, limit, 40.0):
            u = torch.full_like(gate, up)
            g = torch.minimum(gate, torch.tensor(limit).double())
            want = g / (1 + torch.exp(-1.702 * g)) * (min(max(up, -limit), limit) + 1)
            assert torch.allclose(glu.apply(gate, u, glu.ClampedGLU(limit)), want)
            assert torch.allclose(oracle.clamped_glu(gate, u, limit), want)
    with pytest.raises(ValueError):
        glu.ClampedGLU(0.0)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("d", [8, 64, 136])
@pytest.mark.parametrize("limit", [0.4, 1.5])
def test_clamped_activation_kernels(d, limit, kind):
    x, x64 = randn(33, 2 * d, seed=1, kind=kind, scale=3.0)
    act = glu.ClampedGLU(limit)
    near(ops.act_and_mul(x, act), oracle.clamped_glu(x64[:, :d], x64[:, d:], limit), kind)
    if kind[1] == torch.bfloat16 and d % 64 == 0:
        from xllm_b200.ops.gemm_tcgen05 import act_and_mul_interleaved, gemm_act_mul, interleave_gate_up
        il = interleave_gate_up(x[:, :d].T.contiguous(), x[:, d:].T.contiguous()).T.contiguous()
        near(act_and_mul_interleaved(il, act), oracle.clamped_glu(x64[:, :d], x64[:, d:], limit), kind)
        h, h64 = randn(600, 72, seed=2, kind=kind)
        w, w64 = randn(2 * 128, 72, seed=3, kind=kind, scale=0.2)
        got = gemm_act_mul(h, interleave_gate_up(w[:128], w[128:]), act)
        near(got, oracle.clamped_glu(h64 @ w64[:128].T, h64 @ w64[128:].T, limit), kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("T,W,E,top,ff,sff,limits", [(1, 64, 4, 1, 64, 64, (1.0, 0.5)), (40, 128, 8, 2, 64, 192, (0.7, 1.5)),
                                                     (530, 128, 16, 4, 128, 128, (1.5, 1.0)), (19, 72, 5, 3, 20, 12, (1.2, 0.9)),
                                                     (33, 100, 3, 3, 10, 30, (1.0, 1.0))])
def test_expert_layer(T, W, E, top, ff, sff, limits, kind):
    """A mixture of clamped experts with a shared one of another size and limit, through the layer that models use."""
    from xllm_b200.models import ModelArgs
    from xllm_b200.models.qwen_moe import SparseMoeBlock
    dev, dt = kind
    up = lambda n: (n + 63) // 64 * 64 if dt == torch.bfloat16 else n
    args = ModelArgs(num_experts=E, num_experts_per_tok=top, hidden_size=W, moe_intermediate_size=up(ff), scoring_func="softmax",
                     norm_topk_prob=True, n_shared_experts=1, shared_expert_intermediate_size=up(sff))
    block = SparseMoeBlock(args, dt, dev, own_router=False, act=glu.ClampedGLU(limits[0]), shared_act=glu.ClampedGLU(limits[1]))
    load, w64 = dict(block.named_loaders()), {}
    seed = 100
    for name, n, to in [(f"e{e}", ff, f"experts.{e}") for e in range(E)] + [("shared", sff, "shared_experts")]:
        for leaf, shape in (("gate", (n, W)), ("up", (n, W)), ("down", (W, n))):
            seed += 1
            t, w64[f"{name}.{leaf}"] = randn(*shape, seed=seed, kind=("cpu", dt), scale=1.5 * shape[1] ** -0.5)
            extra = up(n) - n
            pad = (0, extra) if leaf == "down" else (0, 0, 0, extra)
            load[f"{to}.{leaf}_proj.weight"](torch.nn.functional.pad(t, pad))
    h, h64 = randn(T, W, seed=5, kind=kind)
    z = torch.randn(T, E, generator=gen(6)).double() * 2
    order = z.argsort(dim=1, descending=True)
    z.scatter_add_(1, order[:, :top], torch.full((T, top), 0.2, dtype=torch.float64))     # no close calls
    got = block(h, logits=z.float().to(dev))
    ids, weights = oracle.route(z, top)
    want = oracle.expert(h64, oracle._sub(w64, "shared."), limits[1])
    for t in range(T):
        for j in range(top):
            want[t] += weights[t, j] * oracle.expert(h64[t:t + 1], oracle._sub(w64, f"e{int(ids[t, j])}."), limits[0])[0]
    near(got, want, kind, loose=0.02)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("E,top", [(8, 2), (5, 1), (64, 6), (3, 3)])
def test_router_weights_are_a_softmax_over_the_chosen(E, top, kind):
    z, z64 = randn(50, E, seed=E, kind=(kind[0], torch.float32), scale=3.0)
    z[0], z64[0] = z[0] * 30, z64[0] * 30                             # far apart: the others' weights underflow to zero
    ids, w = moe_ops.route_reference(z.cpu(), top)
    want_ids, want_w = oracle.route(z64, top)
    assert torch.equal(ids, want_ids) and float((w.double() - want_w).abs().max()) < 1e-6


# ------------------------------------------------------------------------------------------- residual
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("T,W", [(1, 64), (37, 256), (5, 4096), (9, 72), (6, 100), (3, 8192)])
@pytest.mark.parametrize("two", [False, True])
def test_residual_update_with_a_normed_sum(T, W, two, kind):
    """x <- x + norm(half the sum of two normed branches), then the next norm, in one launch."""
    x0 = torch.randn(T, W, generator=gen(1))
    a, a64 = randn(T, W, seed=2, kind=kind)
    b, b64 = randn(T, W, seed=3, kind=kind, scale=5.0)
    ws = [randn(W, seed=4 + i, kind=kind) for i in range(4)]
    (wa, wa64), (wb, wb64), (wsum, wsum64), (wo, wo64) = ws
    x = x0.to(kind[0]).clone()
    kw = dict(y2=b, w2=wb) if two else {}
    _, h = residual_update(x, a, w=wa, coef=0.5, w_sum=wsum, w_out=wo, eps=1e-5, **kw)
    y = oracle.rms_norm(a64, wa64, 1e-5) + (oracle.rms_norm(b64, wb64, 1e-5) if two else 0)
    want = x0.double() + oracle.rms_norm(0.5 * y, wsum64, 1e-5)
    near(x, want, (kind[0], torch.float32))
    near(h, oracle.rms_norm(want, wo64, 1e-5), kind)


def test_oracle_window_counts():
    """The mask of the plain implementation, spelled out."""
    m = oracle.visible(12, 4, 2)
    for i in range(12):
        for j in range(12):
            assert bool(m[i, j]) == (j <= i and (i - j < 4 or j < 2))
    assert math.isclose(float(oracle.rotate(torch.ones(3, 1, 4, dtype=torch.float64), {"dims": 2, "base": 10.0, "scaling": {"factor": 4.0}})
                              [2, 0, 0]), math.cos(0.5) - math.sin(0.5))
