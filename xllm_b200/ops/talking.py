"""Attention whose heads' softmax weights are mixed before they meet the values ("talking heads" behind the softmax), and what lies
between its projections and the cache: a short convolution, norms of whole rows, unit-norm values."""
from __future__ import annotations

import torch

from . import _lib, reference
from ._lib import F, I, L, P, check, ptr, stream

_lib.register_signature("xllm_conv_row_norm_kv", [P, P, P, L, P, P, P, P] + [I] * 7 + [F] + [P] * 7 + [I] * 4 + [P])
_lib.register_signature("xllm_talk_decode", [P, P, P, P, P, P, I, P, I, I, I, I, I, F, F, L, I, I, P, P])
_lib.register_signature("xllm_talk_decode_workspace", [L, I, L, I, I], L)
_lib.register_signature("xllm_prefill_lse_tc", [P, P, L, L, P, L, P, I, P, P, I, I, I, I, I, F, F, P])
_lib.register_signature("xllm_talk_weights", [P, L, L, P, L, P, L, P, P, P, I, P, P, I, I, I, I, I, I, I, F, F, I, P])
_lib.register_signature("xllm_talk_error_status", [])
_lib.register_signature("xllm_talk_values_tc", [P, I, P, L, L, P, L, P, I, P, P, I, I, I, I, I, I, I, P])
_lib.register_signature("xllm_talk_attn_generic", [P, P, P, P, P, P, L, P, I, P, P] + [I] * 9 + [F, F, I, P])

_DT = {torch.bfloat16: 0, torch.float32: 1}

WORKSPACE_BYTES = 1 << 30              # of a chunk of rows
TC_HEAD = 128                        # head size of the tensor-core kernels' caches


def conv_row_norm_kv_write(q, k, v, heads, kv_heads, d, slots, k_cache, v_cache, q_w, k_w, conv, eps=1e-6, long_portions=True):
    """A causal convolution per channel, then an RMS norm of all of q and of all of k with weights [heads * d], [kv_heads * d], and
    every value head over its own root mean square; k and v rows go to the paged caches, whose heads may be wider (zero filled).
    q, k, v: column blocks of the same rows; conv as in ops.rope_norm_kv_write.  Returns q [T, heads, cache head size]."""
    T, dp = q.shape[0], k_cache.shape[3]
    dv = v.shape[1] // kv_heads
    cw, ring, st, cu, kl = conv
    if not q.is_cuda:
        y = reference.conv_portions(torch.cat([q, k, v], dim=1), *conv)
        q, k, v = y.split([q.shape[1], k.shape[1], v.shape[1]], dim=1)
        norm = lambda x: x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
        pad = lambda x: torch.nn.functional.pad(x, (0, dp - x.shape[-1])).to(k_cache.dtype)
        reference.write_kv_cache(pad((norm(k) * k_w.float()).view(T, kv_heads, d)), pad(norm(v.reshape(T, kv_heads, dv))), k_cache,
                                 v_cache, slots)
        return pad((norm(q) * q_w.float()).view(T, heads, d))
    from . import _count, _index
    assert q.stride(0) == k.stride(0) == v.stride(0) and q.stride(1) == k.stride(1) == v.stride(1) == 1
    assert q.dtype == k_cache.dtype == cw.dtype == ring.dtype and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert cw.is_contiguous() and ring.is_contiguous() and ring.shape[1:] == cw.shape
    assert cw.shape[1] == q.shape[1] + k.shape[1] + v.shape[1] and q_w.numel() == q.shape[1] and k_w.numel() == k.shape[1]
    assert st.dtype == cu.dtype == kl.dtype == torch.int32 and cu.shape[0] > st.shape[0] and kl.shape[0] >= st.shape[0]
    slots = _index(slots, torch.int32, "conv_row_norm_kv_write slots")
    out = torch.empty((T, heads, dp), dtype=q.dtype, device=q.device)
    check(_lib.load().xllm_conv_row_norm_kv(
        ptr(q), ptr(k), ptr(v), q.stride(0), ptr(out), ptr(k_cache), ptr(v_cache), ptr(slots), T, heads, kv_heads, d, dv, dp,
        k_cache.shape[2], float(eps), ptr(q_w), ptr(k_w), ptr(cw), ptr(ring), ptr(st), ptr(cu), ptr(kl), st.shape[0], cw.shape[0],
        int(long_portions), _DT[q.dtype], stream()), "conv_row_norm_kv")
    _count(2 if long_portions and cw.shape[0] > 1 else 1)
    return out


def reference_attention(q, k_cache, v_cache, block_table, cu_q, kv_lens, scale, softcap, talk, dv, out):
    """Tensor operations of the same sums, sequence by sequence."""
    nq, nkv, d = q.shape[1], k_cache.shape[1], q.shape[2]
    for b in range(len(kv_lens)):
        qs, qe, kl = int(cu_q[b]), int(cu_q[b + 1]), int(kv_lens[b])
        if qe == qs or kl == 0:
            continue
        k = reference._gather_kv(k_cache, block_table[b], kl).float().repeat_interleave(nq // nkv, dim=0)
        v = reference._gather_kv(v_cache, block_table[b], kl)[..., :dv].float().repeat_interleave(nq // nkv, dim=0)
        s = torch.einsum("qhd,hkd->hqk", q[qs:qe].float(), k) * scale
        if softcap:
            s = softcap * torch.tanh(s / softcap)
        place = torch.arange(qe - qs)[:, None] + (kl - (qe - qs))
        s = s.masked_fill(torch.arange(kl)[None] > place, float("-inf"))
        w = torch.einsum("hg,gqk->hqk", talk.float(), torch.softmax(s, dim=-1))
        out[qs:qe] = torch.einsum("hqk,hkd->qhd", w, v).to(out.dtype)
    return out


def head_size(d, dv, dtype, device):
    """Head size of the paged cache for key heads of d and value heads of dv."""
    n = max(d, dv)
    if dtype == torch.bfloat16 and torch.device(device).type == "cuda" and n <= TC_HEAD:
        return TC_HEAD
    return (n + 7) // 8 * 8 if dtype == torch.bfloat16 and torch.device(device).type == "cuda" else n


def attention(q, k_cache, v_cache, meta, scale, softcap, talk, dv, out):
    """Rows of q [T, heads, cache head size] of all sequences (meta: decode rows and prompt portions) -> out [T, heads, dv].  Every row
    sees its whole past; softcap > 0: scores become softcap * tanh(score / softcap); the softmax weights are mixed by talk
    [heads, heads], weight_h <- sum_g talk[h, g] weight_g, and head h applies its own to the values of its key/value head."""
    n = meta.n_seqs
    args = (meta.block_table[:n], meta.cu_q[:n + 1], meta.kv_lens[:n], scale, softcap, talk, dv, out)
    if not q.is_cuda:
        return reference_attention(q, k_cache, v_cache, *args)
    longest = meta.max_kv_len if meta.max_kv_len > 0 and not meta.padded else meta.block_table.shape[1] * k_cache.shape[2]
    nd, T, nq, nkv = meta.n_decode, q.shape[0], q.shape[1], k_cache.shape[1]
    if q.dtype != torch.bfloat16 or q.shape[2] != TC_HEAD or nq > 64 or k_cache.shape[2] not in (16, 32, 64, 128):
        return attention_generic(q, k_cache, v_cache, *args, longest)
    if nd > 0:
        decode(q[:nd], k_cache, v_cache, meta.block_table[:nd], meta.kv_lens[:nd], scale, softcap, talk, dv, out[:nd], longest)
    if meta.n_prefill > 0:
        if nq <= 32 and nkv * ((nq // nkv + 3) // 4) <= 8:
            prefill(q, k_cache, v_cache, meta.block_table[nd:n], meta.cu_q[nd:n + 1], meta.kv_lens[nd:n], meta.max_q_len, scale, softcap,
                    talk, dv, out, longest, nd)
        else:
            attention_generic(q, k_cache, v_cache, *args, longest, row0=nd)
    return out


def decode(q, k_cache, v_cache, block_table, seq_lens, scale, softcap, talk, dv, out, longest, splits=None, vsplits=None):
    """One row per sequence, q [B, heads, 128] -> out [B, heads, dv]: capped scores to a table, then the mixture and its product with
    the values; `longest`: no sequence is longer (a captured step knows the limit only)."""
    from . import _count, _index, decode_splits
    B, nq, _ = q.shape
    nkv, page = k_cache.shape[1], k_cache.shape[2]
    assert q.is_contiguous() and out.is_contiguous() and q.dtype == k_cache.dtype == out.dtype == talk.dtype == torch.bfloat16
    assert talk.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert block_table.dtype == torch.int32 and block_table.stride(1) == 1
    seq_lens = _index(seq_lens, torch.int32, "talking decode seq_lens")
    ld = (longest + 63) // 64 * 64
    per = max(1, min(B, WORKSPACE_BYTES // (nq * ld * 4)))
    splits = splits or min(decode_splits(per, nkv, nq // nkv), max(1, longest // 128))
    vsplits = vsplits or min(decode_splits(per, 1, 1), max(1, longest // 128))
    ws = torch.empty(int(_lib.load().xllm_talk_decode_workspace(per, nq, ld, splits, vsplits)), dtype=torch.float32, device=q.device)
    for r in range(0, B, per):
        n = min(per, B - r)
        check(_lib.load().xllm_talk_decode(ptr(out[r:]), ptr(q[r:]), ptr(k_cache), ptr(v_cache), ptr(talk), ptr(block_table[r:]),
                                           block_table.stride(0), ptr(seq_lens[r:]), n, nq, nkv, dv, page, float(scale),
                                           float(softcap or 0.0), ld, splits, vsplits, ptr(ws), stream()), "talk_decode")
        _count(3 if vsplits > 1 else 2)
    return out


def prefill(q, k_cache, v_cache, block_table, cu_q, kv_lens, max_q_len, scale, softcap, talk, dv, out, longest, row0,
            keys=None):
    """Prompt rows [row0, T) of q [T, heads, 128] -> the same rows of out [T, heads, dv]; cu_q holds row numbers of q.  The softmax's
    sums of all rows first, then for a chunk of rows the table of mixed weights and its product with the values.  keys: how many a block of the table takes (a multiple of 128)."""
    from . import _count, _index
    T, nq, _ = q.shape
    B, nkv, page, blocks = kv_lens.shape[0], k_cache.shape[1], k_cache.shape[2], k_cache.shape[0]
    assert q.is_contiguous() and out.is_contiguous() and q.dtype == k_cache.dtype == out.dtype == talk.dtype == torch.bfloat16
    assert talk.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert block_table.dtype == torch.int32 and block_table.stride(1) == 1
    cu_q, kv_lens = _index(cu_q, torch.int32, "talking prefill cu_q"), _index(kv_lens, torch.int32, "talking prefill kv_lens")
    ld, lib, s = (longest + 127) // 128 * 128, _lib.load(), stream()
    lse = torch.empty((T, nq), dtype=torch.float32, device=q.device)
    check(lib.xllm_prefill_lse_tc(ptr(lse), ptr(q), q.stride(0), T, ptr(k_cache), blocks, ptr(block_table), block_table.stride(0), ptr(cu_q),
                                  ptr(kv_lens), B, int(max_q_len), nq, nkv, page, float(scale), float(softcap or 0.0), s), "prefill_lse_tc")
    per = max(128, min(T - row0, WORKSPACE_BYTES // (nq * ld * 2) // 128 * 128))
    # a block takes 16 rows and a range of keys: a few blocks per SM, the long rows first
    tiles = -(-min(per, T - row0) // 16)
    keys = keys or max(128, -(-ld // max(1, 600 // tiles)) // 128 * 128)
    w = torch.empty(nq * per * ld, dtype=torch.bfloat16, device=q.device)
    for r in range(row0, T, per):
        n = min(per, T - r)
        check(lib.xllm_talk_weights(ptr(w), per, ld, ptr(q), T, ptr(k_cache), blocks, ptr(talk), ptr(lse), ptr(block_table), block_table.stride(0),
                                    ptr(cu_q), ptr(kv_lens), B, int(max_q_len), r, n, nq, nkv, page, float(scale), float(softcap or 0.0),
                                    keys, s), "talk_weights")
        check(lib.xllm_talk_values_tc(ptr(out), dv, ptr(w), per, ld, ptr(v_cache), blocks, ptr(block_table), block_table.stride(0), ptr(cu_q),
                                      ptr(kv_lens), B, int(max_q_len), r, n, nq, nkv, page, s), "talk_values_tc")
        _count(2)
    _count()
    return out


def attention_generic(q, k_cache, v_cache, block_table, cu_q, kv_lens, scale, softcap, talk, dv, out, max_kv_len, row0=0, rows=None):
    """Any sizes, bf16 or fp32: three launches for a chunk of rows over a table of their weights."""
    from . import _count, _index
    T, nq, d = q.shape
    rows = T - row0 if rows is None else rows
    assert q.is_contiguous() and out.is_contiguous() and q.dtype == k_cache.dtype == out.dtype == talk.dtype and talk.is_contiguous()
    assert block_table.dtype == torch.int32 and block_table.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    cu_q, kv_lens = _index(cu_q, torch.int32, "talking attention cu_q"), _index(kv_lens, torch.int32, "talking attention kv_lens")
    ld = (max_kv_len + 63) // 64 * 64
    per = max(1, min(rows, WORKSPACE_BYTES // (nq * ld * 4)))
    w = torch.empty(per * nq * ld, dtype=torch.float32, device=q.device)
    for r in range(row0, row0 + rows, per):
        n = min(per, row0 + rows - r)
        check(_lib.load().xllm_talk_attn_generic(
            ptr(out), ptr(q), ptr(k_cache), ptr(v_cache), ptr(talk), ptr(w), ld, ptr(block_table), block_table.stride(0), ptr(cu_q),
            ptr(kv_lens), kv_lens.shape[0], r, n, nq, k_cache.shape[1], d, dv, d, k_cache.shape[2], float(scale),
            float(softcap or 0.0), _DT[q.dtype], stream()), "talk_attn_generic")
        _count(3)
    return out
