"""The fp32 residual stream: branches join it and the next sublayer's input leaves it in one pass
(csrc/kernels/residual.cu), and the token-indexed gated activation of a per-token side input."""
from __future__ import annotations

import torch

from . import _lib
from ._lib import F, I, L, P, check, ptr, stream

_lib.register_signature("xllm_residual_update", [P, P, L, P, P, L, P, P, P, L, P, P, I, I, I, F, F, F, I, P])
_lib.register_signature("xllm_gelu_mul_rows", [P, P, L, P, L, L, P, L, I, I, I, I, P])

_lib.register_signature("xllm_postnorm_update", [P, P, L, P, P, P, L, I, I, F, F, I, P])

_DT = {torch.bfloat16: 0, torch.float32: 1}


def residual_update(x, y, w=None, y2=None, w2=None, coef=1.0, rows=None, w_out=None, eps=1e-6, want_out=True,
                    w_out_offset=0.0, w_sum=None):
    """x <- x + m(coef * (n(y) + n(y2))), n = RMS norm with the branch's weight (w, w2) or the identity without one, m the
    same with w_sum;
    returns (x, out) with out = rmsnorm(x) * (w_out + w_out_offset), or x cast to the branch type when w_out is None (None when
    `want_out` is false).  x is fp32 [T, H] and updated in place; x None starts the stream: x = coef * n(y).
    `rows`: y is a table and row t joins as y[rows[t]] (token embedding)."""
    T = rows.shape[0] if rows is not None else y.shape[0]
    H = y.shape[1]
    init = x is None
    if not y.is_cuda:
        def n(b, wt):
            b = b.float()
            return b if wt is None else b / torch.sqrt(b.pow(2).mean(-1, keepdim=True) + eps) * wt.float()
        add = n(y[rows] if rows is not None else y, w)
        if y2 is not None:
            add = add + n(y2, w2)
        add = n(add * coef, w_sum)
        if init:
            x = add
        else:
            x += add
        out = None
        if want_out:
            out = (x if w_out is None else x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (w_out.float() + w_out_offset)).to(y.dtype)
            if out is x:
                out = x.clone()
        return x, out
    if init:
        x = torch.empty((T, H), dtype=torch.float32, device=y.device)
    assert x.dtype == torch.float32 and x.is_contiguous() and x.shape == (T, H)
    assert y.stride(1) == 1 and (y2 is None or (y2.stride(1) == 1 and y2.dtype == y.dtype))
    assert rows is None or (rows.dtype == torch.int64 and rows.is_contiguous())
    out = torch.empty((T, H), dtype=y.dtype, device=y.device) if want_out else None
    check(_lib.load().xllm_residual_update(
        ptr(x), ptr(y), y.stride(0), ptr(w), ptr(y2), y2.stride(0) if y2 is not None else 0, ptr(w2), ptr(w_sum), ptr(rows), y.shape[0],
        ptr(w_out), ptr(out), T, H, int(init), float(coef), float(eps), float(w_out_offset), _DT[y.dtype], stream()), "residual_update")
    from . import _count
    _count()
    return x, out


def postnorm_update(x, y, w, alpha=1.0, groups=1, w_out=None, eps=1e-6):
    """x <- n(alpha * x + y) * w, n = RMS norm of `groups` equal consecutive parts on their own; returns (x, out) with
    out = x cast to the branch type, or n(x) * w_out.  x is fp32 [T, H] and updated in place."""
    T, H = y.shape
    assert H % groups == 0
    if not y.is_cuda:
        def n(b, wt):
            b = b.view(T, groups, H // groups)
            return (b / torch.sqrt(b.pow(2).mean(-1, keepdim=True) + eps)).view(T, H) * wt.float()
        x.copy_(n(alpha * x + y.float(), w))
        return x, (x.clone() if w_out is None else n(x, w_out)).to(y.dtype)
    assert x.dtype == torch.float32 and x.is_contiguous() and x.shape == (T, H) and y.stride(1) == 1
    out = torch.empty((T, H), dtype=y.dtype, device=y.device)
    check(_lib.load().xllm_postnorm_update(ptr(x), ptr(y), y.stride(0), ptr(w), ptr(w_out), ptr(out), T, H, int(groups), float(alpha),
                                           float(eps), _DT[y.dtype], stream()), "postnorm_update")
    from . import _count
    _count()
    return x, out


def gelu_mul_rows(gate, table, ids, col0, dim, out=None):
    """gelu_tanh(gate[t, :dim]) * table[ids[t], col0 : col0 + dim] -> [T, gate width], zero beyond `dim`."""
    T, width = gate.shape
    if not gate.is_cuda:
        e = table[ids][:, col0:col0 + dim].float()
        y = torch.zeros(T, width, dtype=gate.dtype)
        y[:, :dim] = (torch.nn.functional.gelu(gate[:, :dim].float(), approximate="tanh") * e).to(gate.dtype)
        return y
    assert gate.stride(1) == 1 and table.stride(1) == 1 and ids.dtype == torch.int64 and ids.is_contiguous()
    assert table.dtype == gate.dtype
    if out is None:
        out = torch.empty((T, width), dtype=gate.dtype, device=gate.device)
    check(_lib.load().xllm_gelu_mul_rows(ptr(out), ptr(gate), gate.stride(0), ptr(table), table.stride(0), table.shape[0],
                                         ptr(ids), int(col0), T, int(dim), width, _DT[gate.dtype], stream()), "gelu_mul_rows")
    from . import _count
    _count()
    return out
