"""The mechanisms of Vivazen alone against plain implementations: norm after the sum in groups, convolution + row norms + cache write,
attention with mixed heads, rotated latents with windows, sinks and gates in both forms, frequency scaling, activations."""
import math

import pytest
import torch

import vivazen_oracle as oracle
from test_lukinex_mechanisms import KINDS, Paged, gen, i32, near, randn
from xllm_b200 import ops
from xllm_b200.models.layers import AttentionMetadata
from xllm_b200.ops import mla, talking
from xllm_b200.ops.head_norm import head_gate
from xllm_b200.ops.residual import postnorm_update

GPU16 = ("cuda", torch.bfloat16)


def meta_of(b, padded=0, longest=None):
    nd = b.n_decode
    return AttentionMetadata(n_decode=nd, n_prefill=len(b.lens) - nd, slots=b.slots, block_table=b.block_table, kv_lens=b.kv_lens,
                             cu_q=b.cu_q, max_q_len=max(b.new), max_kv_len=max(b.lens) if longest is None else longest,
                             padded=bool(padded))


# ------------------------------------------------------------------------------------------- residual
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("T,W,groups", [(1, 64, 1), (37, 256, 2), (5, 4096, 4), (9, 72, 3), (6, 100, 4), (3, 8192, 1), (130, 96, 12),
                                        (2, 33, 3), (700, 2048, 8)])
@pytest.mark.parametrize("last", [False, True])
def test_norm_after_the_sum(T, W, groups, last, kind):
    """x <- norm(alpha x + y) by parts, and the cast or the next norm of it."""
    x0 = torch.randn(T, W, generator=gen(1)) * torch.linspace(0.2, 4.0, W)    # the parts differ in size
    y, y64 = randn(T, W, seed=2, kind=kind, scale=0.7)
    w, w64 = randn(W, seed=3, kind=kind)
    wo, wo64 = randn(W, seed=4, kind=kind)
    for alpha in (1.0, 2.6, 0.0):
        x = x0.to(kind[0]).clone()
        _, h = postnorm_update(x, y, w, alpha=alpha, groups=groups, w_out=wo if last else None, eps=1e-5)
        want = oracle.join(x0.double(), y64, w64, alpha, groups, 1e-5)
        near(x, want, (kind[0], torch.float32))
        near(h, oracle.grouped_norm(want, wo64, groups, 1e-5) if last else want, kind)


def test_groups_are_normed_apart():
    x = torch.tensor([[3.0, 4.0, 0.3, 0.4]])
    postnorm_update(x, torch.zeros(1, 4), torch.ones(4), alpha=2.0, groups=2, eps=0.0)
    assert torch.allclose(x[0, :2], x[0, 2:]) and abs(float(x[0, 0]) - 3 / math.sqrt(12.5)) < 1e-6


# ------------------------------------------------------------------------------------------- projections to attention
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("heads,kv,d,dv,dp", [(4, 2, 64, 64, 64), (6, 1, 128, 128, 128), (3, 3, 32, 80, 80), (4, 2, 64, 24, 72),
                                              (3, 1, 26, 14, 26), (32, 8, 128, 128, 128), (40, 20, 64, 128, 128)])
def test_convolution_row_norms_and_cache_write(heads, kv, d, dv, dp, taps, kind):
    """Three sequences fed in portions of unequal sizes beside one another, some one token at a time, with other slots and
    padding rows in the batch."""
    dev, dt = kind
    C = heads * d + kv * (d + dv)
    total = [41, 9, 26]
    xs = [randn(n, C, seed=s, kind=kind) for s, n in enumerate(total)]
    cw, cw64 = randn(taps, C, seed=7, kind=kind, scale=0.5)
    qw, qw64 = randn(heads * d, seed=8, kind=kind)
    kw, kw64 = randn(kv * d, seed=9, kind=kind)
    want = []
    for n, (_, x) in zip(total, xs):
        q, k, v = oracle.short_conv(x, cw64.T).split([heads * d, kv * d, kv * dv], dim=1)
        want.append((oracle.rms_norm(q, qw64, 1e-5).view(n, heads, d), oracle.rms_norm(k, kw64, 1e-5).view(n, kv, d),
                     oracle.rms_norm(v.reshape(n, kv, dv), 1.0, 1e-5)))
    ring = torch.full((5, taps, C), float("nan"), dtype=dt, device=dev)
    slot_of = [3, 0, 2]
    kc, vc = (torch.full((12, kv, 16, dp), 9.0, dtype=dt, device=dev) for _ in range(2))
    pages = [[1, 5, 9], [4, 0, 0], [7, 2, 0]]
    at = [0, 0, 0]
    got_q = [[], [], []]
    for sizes in ([1, 5, 0], [2, 1, 3], [1, 1, 1], [13, 0, 7], [1, 2, 2], [23, 0, 13]):
        live = sorted((s for s in range(3) if sizes[s]), key=lambda s: sizes[s] > 1)
        rows, slots, cu = [], [], [0]
        for s in live:
            rows.append(xs[s][0][at[s]:at[s] + sizes[s]])
            slots += [pages[s][p // 16] * 16 + p % 16 for p in range(at[s], at[s] + sizes[s])]
            cu.append(cu[-1] + sizes[s])
        pad = 2                                                       # rows of no sequence
        x = torch.cat(rows + [torch.zeros(pad, C, dtype=dt, device=dev)])
        wide = torch.zeros(x.shape[0], (C + 15) // 8 * 8, dtype=dt, device=dev)   # column blocks of wider rows
        wide[:, :C] = x
        q, k, v = wide[:, :heads * d], wide[:, heads * d:(heads + kv) * d], wide[:, (heads + kv) * d:C]
        conv = (cw, ring, i32([slot_of[s] for s in live], kind), i32(cu, kind), i32([at[s] + sizes[s] for s in live], kind))
        out = talking.conv_row_norm_kv_write(q, k, v, heads, kv, d, i32(slots + [-1] * pad, kind), kc, vc, qw, kw, conv, eps=1e-5,
                                             long_portions=max(sizes) > 1)
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
    assert bool((kc[3] == 9.0).all())                                 # nobody's page


@pytest.mark.gpu
def test_convolution_of_long_portions():
    """Enough rows for runs of tokens per block, three sequences, a run across their borders."""
    kind, heads, kv, d, taps = GPU16, 8, 2, 128, 3
    C, lens = (heads + 2 * kv) * d, [401, 3, 700]
    T = sum(lens)
    x, x64 = randn(T, C, seed=1, kind=kind)
    cw, cw64 = randn(taps, C, seed=2, kind=kind, scale=0.5)
    one = torch.ones(heads * d, dtype=torch.bfloat16, device="cuda")
    ring = torch.full((4, taps, C), float("nan"), dtype=torch.bfloat16, device="cuda")
    kc, vc = (torch.zeros(T // 16 + 1, kv, 16, d, dtype=torch.bfloat16, device="cuda") for _ in range(2))
    cu = [0, 401, 404, T]
    out = talking.conv_row_norm_kv_write(x[:, :heads * d], x[:, heads * d:(heads + kv) * d], x[:, (heads + kv) * d:], heads, kv, d,
                                         i32(list(range(T)), kind), kc, vc, one, one[:kv * d], (cw, ring, i32([2, 0, 1], kind), i32(cu, kind), i32(lens, kind)))
    y = torch.cat([oracle.short_conv(x64[a:b], cw64.T) for a, b in zip(cu, cu[1:])])
    near(out, oracle.rms_norm(y[:, :heads * d], 1.0, 1e-6).view(T, heads, d), kind)
    flat = lambda c: c.permute(0, 2, 1, 3).reshape(-1, kv, d)[:T]
    near(flat(kc), oracle.rms_norm(y[:, heads * d:(heads + kv) * d], 1.0, 1e-6).view(T, kv, d), kind)
    near(flat(vc), oracle.rms_norm(y[:, (heads + kv) * d:].reshape(T, kv, d), 1.0, 1e-6), kind)
    for s, slot in enumerate([2, 0, 1]):
        for p in range(max(0, lens[s] - taps + 1), lens[s]):
            assert torch.equal(ring[slot, p % taps], x[cu[s] + p])


# ------------------------------------------------------------------------------------------- attention with mixed heads
def talk_case(lens, new, heads, kv, d, dv, kind, cap, scale=None, seed=0, spread=1.5):
    b = Paged(lens, new, kind, seed=seed)
    dp = talking.head_size(d, dv, kind[1], kind[0])
    kc, vc = b.cache(kv, dp), b.cache(kv, dp)
    q, q64 = randn(b.cu[-1], heads, d, seed=1 + seed, kind=kind, scale=spread)
    t, t64 = randn(heads, heads, seed=2 + seed, kind=kind, scale=heads ** -0.5)
    want = torch.zeros(b.cu[-1], heads, dv, dtype=torch.float64)
    scale = d ** -0.5 if scale is None else scale
    for s, (l, n) in enumerate(zip(lens, new)):
        k, k64 = randn(l, kv, d, seed=10 + s + seed, kind=kind)
        v, v64 = randn(l, kv, dv, seed=60 + s + seed, kind=kind)
        b.put(kc, s, torch.nn.functional.pad(k, (0, dp - d)))
        b.put(vc, s, torch.nn.functional.pad(v, (0, dp - dv)))
        full = torch.zeros(l, heads, d, dtype=torch.float64)
        full[l - n:] = q64[b.cu[s]:b.cu[s + 1]]
        want[b.cu[s]:b.cu[s + 1]] = oracle.talking_attention(full, k64, v64, scale, cap, t64)[l - n:]
    for c in (kc, vc):                                                # rows behind a sequence's end are never anything but zeros
        for s, l in enumerate(lens):
            if l % 16:
                c[b.table[s][l // 16], :, l % 16:] = 0.0
        c[0] = 0.0
    return b, torch.nn.functional.pad(q, (0, dp - d)), kc, vc, t, scale, want


TALK_SIZES = [(6, 3, 64, 40), (4, 1, 128, 128), (3, 3, 20, 26), (16, 4, 128, 128), (8, 8, 64, 64), (32, 8, 128, 128), (1, 1, 72, 16),
              (12, 4, 40, 200), (5, 5, 128, 128), (24, 2, 128, 128), (64, 8, 128, 128)]


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,kv,d,dv", TALK_SIZES)
def test_talking_attention(heads, kv, d, dv, kind):
    """Decoding and prompt portions over shuffled pages; pages that nobody may read hold NaN."""
    lens, new = [190, 1, 33, 300, 161, 90, 2], [1, 1, 1, 300, 60, 2, 2]
    for cap in (3.0, 50.0):
        b, q, kc, vc, t, scale, want = talk_case(lens, new, heads, kv, d, dv, kind, cap)
        out = torch.zeros(b.cu[-1], heads, dv, dtype=kind[1], device=kind[0])
        talking.attention(q, kc, vc, meta_of(b), scale, cap, t, dv, out)
        near(out, want, kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,kv,d", [(8, 2, 128), (4, 2, 64)])
def test_talking_attention_of_strangers(heads, kv, d, kind):
    """One head sees nothing but a far key, and only another head's mixture lets it through: a lost key, a mixture that is left out
    or transposed, or weights mixed before they are normed would show."""
    for l, far in ((400, 0), (400, 255), (400, 256), (257, 127), (130, 64), (64, 15)):
        for n in (1, 2, 40):
            b = Paged([l], [n], kind)
            kc, vc = b.cache(kv, d, 0.0), b.cache(kv, d, 0.0)
            k = torch.zeros(l, kv, d)
            v = torch.randn(l, kv, d, generator=gen(3)) * 0.05
            k[far, 0, 3] = 8.0
            v[far] = 1.0 + torch.arange(d) / d
            b.put(kc, 0, k)
            b.put(vc, 0, v)
            q = torch.zeros(n, heads, d)
            q[:, 1, 3] = 8.0
            t = torch.zeros(heads, heads)
            t[heads - 1, 1], t[0, 0] = -1.5, 1.0
            q, t = q.to(kc), t.to(kc)
            out = torch.zeros(n, heads, d, dtype=kind[1], device=kind[0])
            talking.attention(q, kc, vc, meta_of(b), 0.5, 30.0, t, d, out)
            full = torch.zeros(l, heads, d, dtype=torch.float64)
            full[l - n:] = q.double().cpu()
            want = oracle.talking_attention(full, k.to(kind[1]).double(), v.to(kind[1]).double(), 0.5, 30.0, t.double().cpu())[l - n:]
            near(out, want, kind)
            if far <= l - n:
                assert float(want[:, heads - 1].abs().min()) > 1.0


@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv,d", [(16, 4, 128), (9, 3, 64)])
def test_talking_attention_in_padded_steps(heads, kv, d):
    """Fixed shapes as a captured step has them: rows and sequences of nobody, and no length known to the host."""
    lens, new = [70, 33, 150, 20], [1, 1, 90, 20]
    b, q, kc, vc, t, scale, want = talk_case(lens, new, heads, kv, d, d, GPU16, 20.0)
    T = b.cu[-1]
    rows = lambda x, n: torch.cat([x, torch.zeros(n, *x.shape[1:], dtype=x.dtype, device=x.device)])
    q2 = torch.cat([q[:2], q[:2] * 0, q[2:], q[:5] * 0])              # two decode rows and five prompt rows of nobody
    m = AttentionMetadata(n_decode=4, n_prefill=4, slots=None, block_table=rows(torch.cat([b.block_table[:2], b.block_table[:2] * 0, b.block_table[2:]]), 2),
                          kv_lens=i32([70, 33, 0, 0, 150, 20, 0, 0], GPU16), cu_q=i32([0, 1, 2, 3, 4, 94, 114, 114, 114], GPU16),
                          max_q_len=115, max_kv_len=0, padded=True)
    out = torch.zeros(T + 7, heads, d, dtype=torch.bfloat16, device="cuda")
    talking.attention(q2, kc, vc, m, scale, 20.0, t, d, out)
    near(torch.cat([out[:2], out[4:T + 2]]), want, GPU16)
    assert bool(torch.isfinite(out).all())


@pytest.mark.gpu
def test_talking_attention_in_chunks_of_rows(monkeypatch):
    """A workspace for a few rows at a time gives the same answers."""
    for heads, kv, d in ((4, 2, 40), (16, 4, 128)):
        b, q, kc, vc, t, scale, want = talk_case([200, 300, 180], [1, 300, 70], heads, kv, d, d, GPU16, 20.0)
        monkeypatch.setattr(talking, "WORKSPACE_BYTES", heads * 320 * 4 * 100)
        out = torch.zeros(b.cu[-1], heads, d, dtype=torch.bfloat16, device="cuda")
        talking.attention(q, kc, vc, meta_of(b), scale, 20.0, t, d, out)
        near(out, want, GPU16)


@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv,d,dv", [(32, 8, 128, 128), (20, 1, 128, 72), (12, 4, 64, 40), (7, 7, 128, 96), (2, 1, 32, 128)])
def test_talking_decode_in_splits(heads, kv, d, dv):
    """Any cut of the context for the scores and for the values, empty shares included."""
    lens = [1290, 1, 64, 65, 700, 128]
    b, q, kc, vc, t, scale, want = talk_case(lens, [1] * 6, heads, kv, d, dv, GPU16, 20.0)
    for splits, vsplits in ((None, None), (1, 1), (3, 1), (1, 5), (9, 16), (16, 30)):
        out = torch.zeros(6, heads, dv, dtype=torch.bfloat16, device="cuda")
        talking.decode(q, kc, vc, b.block_table, b.kv_lens, scale, 20.0, t, dv, out, max(lens), splits=splits, vsplits=vsplits)
        near(out, want, GPU16)


@pytest.mark.gpu
@pytest.mark.parametrize("heads,kv,d,dv", [(32, 8, 128, 128), (12, 4, 64, 40), (5, 5, 128, 96), (3, 1, 32, 128)])
@pytest.mark.parametrize("cap,spread", [(30.0, 1.0), (6.0, 4.0), (300.0, 2.0), (0.0, 1.0)])
def test_talking_prompts_of_many_key_tiles(heads, kv, d, dv, cap, spread):
    """Blocks that walk over several tiles of keys; scores within the polynomial's reach, beyond it, under a cap too high for sums
    without a reference, and without a cap; portions behind long contexts."""
    lens, new = [700, 1290, 513], [700, 90, 17]
    b, q, kc, vc, t, scale, want = talk_case(lens, new, heads, kv, d, dv, GPU16, cap or 1e6, spread=spread)
    for keys in (128, 384, 1408):
        out = torch.zeros(b.cu[-1], heads, dv, dtype=torch.bfloat16, device="cuda")
        talking.prefill(q, kc, vc, b.block_table, b.cu_q, b.kv_lens, max(new), scale, cap, t, dv, out, max(lens), 0, keys=keys)
        near(out, want, GPU16)
    assert ops._lib.load().xllm_talk_error_status() == 0 and ops._lib.load().xllm_fmha_error_status() == 0


# ------------------------------------------------------------------------------------------- latent attention
ROTS = [dict(base=10000.0, dims=16, scaling=dict(factor=3.0, original=64, fast=8.0, slow=0.5)),
        dict(base=500.0, dims=32, scaling=dict(factor=1.0, original=2048, fast=32.0, slow=1.0)),
        dict(base=1e6, dims=64, scaling=dict(factor=40.0, original=4096, fast=32.0, slow=1.0)),
        dict(base=50.0, dims=2, scaling=dict(factor=2.0, original=100, fast=4.0, slow=2.0)),
        dict(base=300.0, dims=10, scaling=dict(factor=8.0, original=32, fast=1.0, slow=1.0))]


def table(rot, n, device):
    s = rot["scaling"]
    return ops.reference.build_cos_sin_cache(rot["dims"], n, rot["base"],
                                             {"rope_type": "yarn", "factor": s["factor"], "original_max_position_embeddings": s["original"],
                                              "beta_fast": s["fast"], "beta_slow": s["slow"],
                                              "attention_factor": 0.1 * math.log(s["factor"]) + 1.0}, device)


@pytest.mark.parametrize("rot", ROTS)
def test_scaled_frequencies(rot):
    cs, half = table(rot, 700, "cpu").double(), rot["dims"] // 2
    freq, size = oracle.yarn_frequencies(rot)
    for p in (0, 1, 63, 64, 699):
        for i, f in enumerate(freq):
            assert abs(float(cs[p, i]) - size * math.cos(p * f)) < 1e-6 and abs(float(cs[p, half + i]) - size * math.sin(p * f)) < 1e-6


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,d,rank,rot", [(3, 24, 40, ROTS[0]), (5, 32, 88, ROTS[1]), (4, 64, 448, ROTS[2]), (2, 128, 512, ROTS[2]),
                                              (5, 7, 33, ROTS[3]), (2, 20, 520, ROTS[4]), (16, 96, 300, ROTS[1])])
def test_latent_rows_and_rotation(heads, d, rank, rot, kind):
    """Normed latents and the rotated key part in the cache rows, queries turned in place and beside their absorbed form."""
    dev, dt = kind
    r, T, pos = rot["dims"], 9, [0, 1, 2, 63, 64, 65, 5, 300, 699]
    width, at, _ = mla.row_layout(rank, r, dt, dev)
    hs = d + r + 4
    ld = (heads * hs + 7) // 8 * 8 + (rank + r + 7) // 8 * 8
    rows, r64 = randn(T, ld, seed=1, kind=kind)
    c0 = (heads * hs + 7) // 8 * 8
    w, w64 = randn(rank, seed=2, kind=kind)
    cache = torch.full((4, 1, 16, width), 7.0, dtype=dt, device=dev)
    slots = [17, 16, -1, 40, 63, 18, 5, 0, 33]
    qa = torch.full((T, heads, width), 3.0, dtype=dt, device=dev)
    mla.rope_write(rows[:, :heads * hs], heads, d, rows[:, c0:c0 + rank + r], w, rank, r, at, table(rot, 700, dev),
                   torch.tensor(pos, device=dev), i32(slots, kind), cache, 1e-5, qa=qa, qa_rows=5)
    turn = lambda x, p: oracle.rotate_pairs(x.view(1, -1, r), rot, p)[0]
    q = r64[:, :heads * hs].reshape(T, heads, hs).clone()
    for t, p in enumerate(pos):
        q[t, :, d:d + r] = turn(q[t, :, d:d + r].contiguous(), p)
    near(rows[:, :heads * hs].reshape(T, heads, hs), q, kind)
    near(qa[:5, :, at:at + r], q[:5, :, d:d + r], kind)
    assert bool((qa[:, :, :rank] == 3.0).all()) and bool((qa[5:] == 3.0).all())
    assert not bool(qa[:5, :, rank:at].any()) and not bool(qa[:5, :, at + r:].any())
    flat = cache.view(-1, width)
    for t, s in enumerate(slots):
        if s >= 0:
            near(flat[s, :rank], oracle.rms_norm(r64[t, c0:c0 + rank], w64, 1e-5), kind)
            near(flat[s, at:at + r], turn(r64[t, c0 + rank:c0 + rank + r], pos[t])[0], kind)
            assert not bool(flat[s, rank:at].any()) and not bool(flat[s, at + r:].any())
    assert bool((flat[[s for s in range(64) if s not in slots]] == 7.0).all())


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("d,heads,kv", [(64, 6, 3), (128, 4, 1), (256, 2, 1), (72, 3, 3)])
@pytest.mark.parametrize("window", [0, 1, 20, 64, 130])
def test_sinks(d, heads, kv, window, kind):
    """Prompt portions with sinks far below, among and far above the scores; windows and pages that were given back."""
    lens, new = [190, 300, 161, 90], [1, 300, 60, 2]
    b = Paged(lens, new, kind)
    kc, vc = b.cache(kv, d), b.cache(kv, d)
    q, q64 = randn(b.cu[-1], heads, d, seed=1, kind=kind, scale=1.5)
    sink = torch.tensor([-30.0, 1.5, 9.0, 3.0, 0.0, 40.0])[:heads]
    want = torch.zeros(b.cu[-1], heads, d, dtype=torch.float64)
    for s, (l, n) in enumerate(zip(lens, new)):
        k, k64 = randn(l, kv, d, seed=10 + s, kind=kind)
        v, v64 = randn(l, kv, d, seed=20 + s, kind=kind)
        b.put(kc, s, k)
        b.put(vc, s, v)
        full = torch.zeros(l, heads, d, dtype=torch.float64)
        full[l - n:] = q64[b.cu[s]:b.cu[s + 1]]
        each = lambda x: x.repeat_interleave(heads // kv, dim=1)
        want[b.cu[s]:b.cu[s + 1]] = oracle.sink_attention(full, each(k64), each(v64), d ** -0.5, oracle.visible(l, window or None),
                                                          sink.double())[l - n:]
        for p in range(max(0, l - n - window + 1) // 16 if window else 0):
            kc[b.table[s][p]] = vc[b.table[s][p]] = float("nan")
            b.block_table[s, p] = 0
    for c in (kc, vc):
        for s, l in enumerate(lens):
            if l % 16:
                c[b.table[s][l // 16], :, l % 16:] = 0.0
        c[0] = 0.0
    out, sink = torch.zeros_like(q), sink.to(kind[0])
    if not q.is_cuda or kind[1] != torch.bfloat16 or d == 72:
        ops.paged_attention_generic(q, kc, vc, b.block_table, b.cu_q, b.kv_lens, d ** -0.5, out=out, window=window, sink=sink)
        near(out, want, kind)
    else:
        ops.paged_prefill_attention(q, kc, vc, b.block_table[1:], b.cu_q[1:], b.kv_lens[1:], max(new), d ** -0.5, out=out,
                                    window=window, sink=sink)
        near(out[1:], want[1:], kind)
    with pytest.raises(TypeError):
        ops._sink(sink.double(), heads, "sinks")


@pytest.mark.gpu
@pytest.mark.parametrize("heads", [1, 7, 16, 33])
@pytest.mark.parametrize("width", mla.LATENT_WIDTHS + (576,))
@pytest.mark.parametrize("window", [0, 1, 17, 64, 300])
def test_latent_decode_with_windows_and_sinks(width, heads, window):
    """One row per sequence and rows of prompt portions, any split of the context; rows in front of every window hold NaN."""
    kind, dv = GPU16, 512 if width == 576 else width
    lens, new = [1, 16, 17, 250, 700, 90], [1, 1, 1, 1, 1, 30]
    b = Paged(lens, new, kind)
    cache = b.cache(1, width, fill=0.0)
    sink = torch.linspace(-3.0, 9.0, heads) if heads > 1 else torch.tensor([2.0])
    q, q64 = randn(b.cu[-1], heads, width, seed=50, kind=kind, scale=1.5)
    want = torch.zeros(b.cu[-1], heads, dv, dtype=torch.float64)
    for s, (l, n) in enumerate(zip(lens, new)):
        c, c64 = randn(l, 1, width, seed=s, kind=kind)
        b.put(cache, s, c)
        full = torch.zeros(l, heads, width, dtype=torch.float64)
        full[l - n:] = q64[b.cu[s]:b.cu[s + 1]]
        each = c64.expand(l, heads, width)
        want[b.cu[s]:b.cu[s + 1]] = oracle.sink_attention(full, each, each[..., :dv], width ** -0.5, oracle.visible(l, window or None),
                                                          sink.double())[l - n:]
        for p in range(max(0, l - n - window + 1) // 16 if window else 0):
            cache[b.table[s][p]] = float("nan")
    nd, sink = b.n_decode, sink.cuda()
    for splits in (None, 1, 2, 5):
        got = mla.latent_decode(q[:nd], cache, b.block_table, width ** -0.5, seq_lens=b.kv_lens[:nd], splits=splits, window=window,
                                sink=sink)
        near(got, want[:nd], kind)
        got = mla.latent_decode(q[nd:], cache, b.block_table, width ** -0.5, positions=b.positions[nd:],
                                bt_rows=torch.full((30,), 5, dtype=torch.int32, device="cuda"), splits=splits, window=window, sink=sink)
        near(got, want[nd:], kind)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,dv,dp", [(3, 20, 26), (8, 128, 128), (6, 40, 128), (1, 16, 16)])
def test_gate_per_head(heads, dv, dp, kind):
    a, a64 = randn(9, heads, dp, seed=1, kind=kind)
    g, g64 = randn(9, heads + 3, seed=2, kind=kind, scale=2.0)
    got = head_gate(a, g[:, :heads], dv)
    near(got, (a64[..., :dv] / (1 + torch.exp(-g64[:, :heads, None]))).reshape(9, -1), kind)


class Owner:
    """A LatentAttention with random weights and the projection rows it asks for."""

    def __init__(self, W, heads, d, dv, rank, rot, window, kind, seed=0):
        from xllm_b200.models.layers import RotaryEmbedding
        from xllm_b200.models.mixers import FusedProjection, LatentAttention
        dev, dt = kind
        s = rot["scaling"]
        rope = RotaryEmbedding(rot["dims"], 2048, rot["base"],
                               {"rope_type": "yarn", "factor": s["factor"], "original_max_position_embeddings": s["original"],
                                "beta_fast": s["fast"], "beta_slow": s["slow"],
                                "attention_factor": 0.1 * math.log(s["factor"]) + 1.0}, dev, interleaved=True)
        self.cfg = dict(heads=heads, dim=d, vdim=dv, kv_rank=rank, rot_dim=rot["dims"], rot=rot, scale=(d + rot["dims"]) ** -0.5,
                        mask=dict(size=window))
        self.mix = LatentAttention(W, heads, d, dv, 0, rank, self.cfg["scale"], 1e-5, dt, dev, rope=rope, window=window, sink=True,
                                   gate=True)
        self.proj = self.mix.add_module("in", FusedProjection(W, self.mix.width_parts(), dt, dev))
        shapes = oracle.tensor_shapes({"width": W, "vocab": 1, "layers": [{"type": "latent_attention", "mixer": self.cfg, "mlp": None}]})
        w = {n: torch.randn(sh, generator=gen(seed + i)) * (sh[-1] ** -0.5 if len(sh) > 1 else 1.0) for i, (n, sh) in enumerate(shapes.items())}
        self.w = {n[len("l0.mix."):]: t.to(dt) for n, t in w.items() if n.startswith("l0.mix.")}
        self.mix.load_weights((n + (".weight" if n == "o" else ""), t) for n, t in self.w.items())

    def want(self, x64):
        return oracle.latent_mixer(x64, {n: t.double() for n, t in self.w.items()}, self.cfg, 1e-5)


@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("heads,d,dv,rank,rot,window", [(3, 24, 20, 40, ROTS[0], 33), (4, 64, 128, 448, ROTS[2], 100),
                                                        (8, 96, 80, 200, ROTS[1], 64), (2, 40, 64, 512, ROTS[2], 300),
                                                        (2, 128, 128, 300, ROTS[2], 50), (5, 30, 33, 50, ROTS[4], 7)])
def test_latent_attention_in_portions(heads, d, dv, rank, rot, window, kind):
    """One sequence through the mixer in portions, large (expanded on the tensor cores where the sizes allow) and small."""
    W, n = 64, 700 if kind[0] == "cuda" else 150
    o = Owner(W, heads, d, dv, rank, rot, window, kind)
    x, x64 = randn(n, W, seed=9, kind=kind)
    want = o.want(x64)
    calls, plain = [], ops.ragged_prefill_attention
    ops.ragged_prefill_attention = lambda *a, **k: (calls.append(1), plain(*a, **k))[1]
    try:
        for cuts in ([n], [90, 1, 300, 2, 1], [n - 2, 2], [n - 1, 1]):
            b = Paged([n], [n], kind)
            cache = torch.zeros(b.blocks, 1, 16, o.mix.width, dtype=kind[1], device=kind[0])
            got, at, i = [], 0, 0
            while at < n:
                m = min(cuts[i % len(cuts)], n - at)
                nd = int(m == 1)
                meta = AttentionMetadata(n_decode=nd, n_prefill=1 - nd, slots=b.slots[at:at + m], block_table=b.block_table,
                                         kv_lens=i32([at + m], kind), cu_q=i32([0, m], kind), max_q_len=m, max_kv_len=at + m)
                got.append(o.mix(o.proj, o.proj(x[at:at + m]), b.positions[at:at + m], meta, (cache, cache), None))
                at, i = at + m, i + 1
            near(torch.cat(got), want, kind, loose=0.03)
    finally:
        ops.ragged_prefill_attention = plain
    assert bool(calls) == (o.mix.expand_from is not None)


# ------------------------------------------------------------------------------------------- activation
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("d", [8, 64, 136])
def test_gelu_gate(d, kind):
    x, x64 = randn(33, 2 * d, seed=1, kind=kind, scale=2.0)
    near(ops.act_and_mul(x, "gelu_tanh"), oracle.gelu_tanh(x64[:, :d]) * x64[:, d:], kind)


def test_oracle_masks_and_frequencies():
    m = oracle.visible(9, 4)
    assert all(bool(m[i, j]) == (0 <= i - j < 4) for i in range(9) for j in range(9))
    rot = dict(base=100.0, dims=4, scaling=dict(factor=4.0, original=1000, fast=1e6, slow=1e-6))
    f, size = oracle.yarn_frequencies(rot)                            # between the ramp's ends: the share follows the pair
    lo, hi = 0, 3
    assert math.isclose(f[1], 100.0 ** -0.5 * (1 / 3 / 4 + 2 / 3)) and math.isclose(size, 1 + 0.1 * math.log(4.0)) and f[0] == 1.0
    p = oracle.softmax(torch.tensor([[0.0, 1.0]]).double(), torch.tensor([[True, True]]), torch.tensor(2.0).double())
    e = [1.0, math.e, math.e ** 2]
    assert abs(float(p[0, 1]) - e[1] / sum(e)) < 1e-12
