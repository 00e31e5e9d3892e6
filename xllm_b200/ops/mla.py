"""Front end of the MLA kernels (`csrc/kernels/mla.cu`): latent-cache write + rotary embeddings, and
absorbed multi-head latent attention over the paged latent cache.  CPU tensors take the PyTorch
reference of the same math."""
from __future__ import annotations

import torch

from . import _lib
from ._lib import F, I, L, P, check, ptr, stream

_lib.register_signature("xllm_mla_decode", [P, P, L, P, P, I, P, P, P, I, I, I, F, I, P, P])
_lib.register_signature("xllm_mla_cache_write", [P, L, P, F, P, P, P, P, P, L, L, P, I, I, P])
_lib.register_signature("xllm_mla_decode_workspace", [L, I, I], L)

LATENT, ROT = 512, 64


def rope_pairs(v, cos_sin_rows):
    """Rotary embedding on adjacent pairs of the last dimension; cos_sin_rows [T, rot] = cos | sin."""
    half = v.shape[-1] // 2
    cs = cos_sin_rows.float()
    shape = [cs.shape[0]] + [1] * (v.dim() - 2) + [half]
    cos, sin = cs[:, :half].reshape(shape), cs[:, half:].reshape(shape)
    vf = v.float()
    x1, x2 = vf[..., 0::2], vf[..., 1::2]
    return torch.stack([x1 * cos - x2 * sin, x2 * cos + x1 * sin], dim=-1).flatten(-2).to(v.dtype)


def cache_write(kv_a, norm_w, eps, cos_sin, positions, slots, cache, q_rope, q_cat):
    """cache row of every token's slot = [rmsnorm(kv_a[:, :512]) * w | rope(kv_a[:, 512:])];
    q_cat[..., 512:] = rope(q_rope) for every head.  cache: any tensor whose memory is rows of 576."""
    T = kv_a.shape[0]
    # the kernels are built for DeepSeek's widths (512 + 64); anything else (tiny test models) takes
    # the tensor-op form, on whatever device it lives
    if not kv_a.is_cuda or norm_w.shape[0] != LATENT or kv_a.shape[1] != LATENT + ROT:
        from . import reference
        lat = norm_w.shape[0]                      # the reference takes any latent / rotary width
        c, _ = reference.rmsnorm(kv_a[:, :lat].contiguous(), norm_w, eps)
        cs = cos_sin[positions.long()]
        row = torch.cat([c.to(kv_a.dtype), rope_pairs(kv_a[:, lat:], cs)], dim=-1)
        rows = cache.view(-1, kv_a.shape[1])
        if slots is not None:
            ok = slots >= 0
            rows.index_copy_(0, slots[ok].long(), row[ok].to(rows.dtype))
        if q_cat is not None:
            q_cat[..., lat:] = rope_pairs(q_rope, cs)
        return
    assert kv_a.dtype == torch.bfloat16 and kv_a.stride(1) == 1 and kv_a.shape[1] == LATENT + ROT
    assert cos_sin.dtype == torch.float32 and cos_sin.shape[1] == ROT and cache.is_contiguous()
    nh = 0
    if q_cat is not None:
        nh = q_cat.shape[1]
        assert q_cat.is_contiguous() and q_rope.stride(2) == 1 and q_rope.shape[2] == ROT
    check(_lib.load().xllm_mla_cache_write(ptr(kv_a), kv_a.stride(0), ptr(norm_w), float(eps), ptr(cos_sin), ptr(positions),
                                           ptr(slots), ptr(cache), ptr(q_rope) if q_cat is not None else None,
                                           q_rope.stride(0) if q_cat is not None else 0,
                                           q_rope.stride(1) if q_cat is not None else 0, ptr(q_cat), T, nh, stream()),
          "mla_cache_write")
    from . import _count
    _count()


def decode_reference(q_cat, cache, block_table, seq_lens, bt_rows, scale, latent=LATENT):
    rows = cache.view(-1, cache.shape[-1]).float()
    page = cache.shape[-2]
    N, nh, _ = q_cat.shape
    out = torch.zeros(N, nh, latent, dtype=torch.float32, device=q_cat.device)
    for n in range(N):
        sl = int(seq_lens[n])
        if sl <= 0:
            continue
        bt = block_table[int(bt_rows[n]) if bt_rows is not None else n]
        idx = (bt[: (sl + page - 1) // page].long()[:, None] * page + torch.arange(page, device=q_cat.device)).flatten()[:sl]
        ctx = rows[idx]
        s = (q_cat[n].float() @ ctx.T) * scale
        out[n] = torch.softmax(s, dim=-1) @ ctx[:, :latent]
    return out.to(q_cat.dtype)


def decode(q_cat, cache, block_table, scale, seq_lens=None, positions=None, bt_rows=None, splits=None, out=None,
           latent=LATENT):
    """out [N, nh, 512] = absorbed MLA attention of q_cat [N, nh, 576] over the latent cache
    [n_blocks, (1,) page, 576].  Row n sees seq_lens[n] tokens (or positions[n] + 1) of the sequence whose
    block-table row is bt_rows[n] (default n)."""
    N, nh, _ = q_cat.shape
    if not q_cat.is_cuda or latent != LATENT or q_cat.shape[2] != LATENT + ROT:
        lens = seq_lens if seq_lens is not None else positions + 1
        y = decode_reference(q_cat, cache, block_table, lens, bt_rows, scale, latent)
        if out is not None:
            out.copy_(y)
            return out
        return y
    assert q_cat.dtype == torch.bfloat16 and q_cat.stride(2) == 1 and q_cat.stride(1) == LATENT + ROT
    assert cache.is_contiguous() and block_table.dtype == torch.int32
    page = cache.shape[-2]
    if out is None:
        out = torch.empty((N, nh, LATENT), dtype=q_cat.dtype, device=q_cat.device)
    assert out.is_contiguous()
    if N == 0:
        return out
    if splits is None:
        from . import decode_splits
        splits = decode_splits(N, 1, nh)
    ws = None
    if splits > 1:
        ws = torch.empty(int(_lib.load().xllm_mla_decode_workspace(N, nh, splits)), dtype=torch.float32, device=q_cat.device)
    check(_lib.load().xllm_mla_decode(ptr(out), ptr(q_cat), q_cat.stride(0), ptr(cache), ptr(block_table),
                                      block_table.stride(0), ptr(seq_lens), ptr(positions), ptr(bt_rows), N, nh, page,
                                      float(scale), int(splits), ptr(ws), stream()), "mla_decode")
    from . import _count
    _count(2 if splits > 1 else 1)
    return out


# ----------------------------------------------------------------------------- caches of latents alone
_lib.register_signature("xllm_latent_decode", [P, P, L, P, I, P, I, P, P, P, I, I, I, F, I, P, I, P, P])
_lib.register_signature("xllm_latent_norm", [P, P, P, I, I, P, P, P, I, I, P, L, I, F, I, P])
_lib.register_signature("xllm_latent_gather", [P, P, P, I, P, P, P, I, I, I, I, I, P])
_lib.register_signature("xllm_latent_rope_write", [P, I, I, I, P, P, I, I, I, L, P, L, P, P, P, I, P, I, I, F, I, P])

LATENT_WIDTHS = (128, 256, 512)


def latent_width(rank, dtype, device):
    """Row size a cache of latents of `rank` values should have: the widths of the tensor-core kernels in bf16 on the device
    (zero filled), the rank itself otherwise."""
    return row_layout(rank, 0, dtype, device)[0]


def row_layout(rank, rot, dtype, device):
    """(row size, place of the rotated part, how many leading values of a row are value) of a cache of latents with `rot`
    rotated key values beside each."""
    if dtype == torch.bfloat16 and torch.device(device).type == "cuda":
        for w in LATENT_WIDTHS:
            if rank + rot <= w:
                return w, rank, w
        if rank <= LATENT and 0 < rot <= ROT:
            return LATENT + ROT, LATENT, LATENT
        w = (rank + rot + 7) // 8 * 8
        return w, rank, w
    return rank + rot, rank, rank + rot


def rope_write(q, heads, d, c, c_w, rank, rot, rot_at, cos_sin, positions, slots, cache, eps, qa=None, qa_rows=0):
    """Cache row of every token's slot = [rmsnorm(c[:, :rank]) * c_w | rotated c[:, rank:] at rot_at], zeros elsewhere; the part
    [d, d + rot) of every head of q turns in place.  q [T, heads * head stride] and c [T, rank + rot]: column blocks of the same
    rows; neighbouring elements are a pair.  qa [T, heads, width]: absorbed queries, whose first `qa_rows` rows get their columns
    from `rank` on."""
    T, hs, width = q.shape[0], q.shape[1] // heads, cache.shape[-1]
    assert q.stride() == c.stride() and q.stride(1) == 1 and c.shape[1] == rank + rot and cache.is_contiguous()
    if not q.is_cuda:
        cs = cos_sin[positions.long()]
        row = torch.zeros(T, width, dtype=cache.dtype)
        x = c[:, :rank].float()
        row[:, :rank] = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * c_w.float()
        row[:, rot_at:rot_at + rot] = rope_pairs(c[:, rank:], cs)
        ok = slots >= 0
        cache.view(-1, width)[slots[ok].long()] = row[ok]
        part = q.unflatten(1, (heads, hs))[:, :, d:d + rot]
        part.copy_(rope_pairs(part, cs))
        if qa is not None:
            qa[:qa_rows, :, rank:] = 0
            qa[:qa_rows, :, rot_at:rot_at + rot] = part[:qa_rows]
        return
    from . import _count, _index
    assert q.dtype == c.dtype == cache.dtype == c_w.dtype and q.dtype in (torch.bfloat16, torch.float32) and cache.shape[1] == 1
    assert cos_sin.dtype == torch.float32 and cos_sin.shape[1] == rot and cos_sin.is_contiguous()
    assert qa is None or (qa.is_contiguous() and qa.dtype == q.dtype and qa.shape[1:] == (heads, width) and qa.shape[0] >= qa_rows)
    check(_lib.load().xllm_latent_rope_write(
        ptr(q), heads, hs, d, ptr(c), ptr(c_w), rank, rot, rot_at, q.stride(0), ptr(cos_sin), cos_sin.shape[0],
        ptr(_index(positions, torch.int64, "rope_write positions")), ptr(_index(slots, torch.int32, "rope_write slots")), ptr(cache),
        width, ptr(qa), int(qa_rows), T, float(eps), 0 if q.dtype == torch.bfloat16 else 1, stream()), "latent_rope_write")
    _count()


def latent_norm(q, q_w, q_pad, eps, c=None, c_w=None, slots=None, cache=None):
    """Normed query latents [T, q_pad] (zero filled) and, with c, normed latents into the cache rows of the tokens' slots.
    q [T, q rank], c [T, rank]: column blocks of the same rows; cache [n_blocks, 1, page, width]."""
    T, q_rank = q.shape
    out = torch.empty((T, q_pad), dtype=q.dtype, device=q.device)
    if not q.is_cuda:
        def norm(x, w, to):
            x = x.float()
            x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()
            return torch.nn.functional.pad(x, (0, to - x.shape[1])).to(q.dtype)
        out.copy_(norm(q, q_w, q_pad))
        if c is not None:
            ok = slots >= 0
            cache.view(-1, cache.shape[-1])[slots[ok].long()] = norm(c, c_w, cache.shape[-1])[ok]
        return out
    assert q.stride(1) == 1 and q.dtype in (torch.bfloat16, torch.float32)
    if c is not None:
        assert c.stride() == q.stride() and c.dtype == q.dtype == cache.dtype and cache.is_contiguous() and cache.shape[1] == 1
        assert slots.dtype == torch.int32 and slots.is_contiguous()
    check(_lib.load().xllm_latent_norm(ptr(q), ptr(q_w), ptr(out), q_rank, q_pad, ptr(c), ptr(c_w), ptr(cache),
                                       c.shape[1] if c is not None else 0, cache.shape[-1] if c is not None else 0, ptr(slots),
                                       q.stride(0), T, float(eps), 0 if q.dtype == torch.bfloat16 else 1, stream()),
          "latent_norm")
    from . import _count
    _count()
    return out


def latent_decode(q, cache, block_table, scale, seq_lens=None, positions=None, bt_rows=None, splits=None, out=None, window=0,
                  sink=None):
    """`decode` over a cache [n_blocks, 1, page, width]: q [N, nh, width], out the same (512 wide over rows of 576).  CUDA, bf16,
    width in LATENT_WIDTHS or 576.  window > 0: a row sees its last `window` tokens; sink [nh] fp32: exp(sink) joins the denominators."""
    N, nh, width = q.shape
    dv = LATENT if width == LATENT + ROT else width
    assert q.dtype == cache.dtype == torch.bfloat16 and q.is_contiguous() and cache.is_contiguous() and cache.shape[-1] == width
    assert block_table.dtype == torch.int32 and block_table.stride(1) == 1
    if out is None:
        out = torch.empty((N, nh, dv), dtype=q.dtype, device=q.device)
    assert out.is_contiguous() and out.shape == (N, nh, dv)
    if N == 0:
        return out
    from . import _sink
    if splits is None:
        from . import decode_splits
        splits = decode_splits(N, 1, nh)
        if window:
            splits = min(splits, max(1, window // 256))
    ws = torch.empty(N * nh * splits * (dv + 1), dtype=torch.float32, device=q.device) if splits > 1 else None
    check(_lib.load().xllm_latent_decode(ptr(out), ptr(q), q.stride(0), ptr(cache), width, ptr(block_table),
                                         block_table.stride(0), ptr(seq_lens), ptr(positions), ptr(bt_rows), N, nh,
                                         cache.shape[-2], float(scale), int(splits), ptr(ws), int(window), ptr(_sink(sink, nh, "latent_decode")),
                                         stream()), "latent_decode")
    from . import _count
    _count(2 if splits > 1 else 1)
    return out


def latent_gather(cache, block_table, kv_lens, rows_per, cu_q=None, window=0):
    """The cached rows of a few sequences, dense [n_seqs * rows_per, width], zeros behind each sequence.  With a window (and cu_q
    [n_seqs + 1], the rows of the batch) only what these rows see; returns (rows, their number per sequence)."""
    n, width = kv_lens.shape[0], cache.shape[-1]
    assert cache.dtype == torch.bfloat16 and cache.is_contiguous() and cache.shape[1] == 1
    assert block_table.dtype == kv_lens.dtype == torch.int32 and block_table.stride(1) == 1
    assert not window or (cu_q.dtype == torch.int32 and cu_q.is_contiguous())
    out = torch.empty((n * rows_per, width), dtype=cache.dtype, device=cache.device)
    lens = torch.empty(n, dtype=torch.int32, device=cache.device) if window else None
    check(_lib.load().xllm_latent_gather(ptr(out), ptr(cache), ptr(block_table), block_table.stride(0), ptr(kv_lens),
                                         ptr(cu_q), ptr(lens), int(window), n, rows_per, cache.shape[-2], width, stream()),
          "latent_gather")
    from . import _count
    _count()
    return (out, lens) if window else out
