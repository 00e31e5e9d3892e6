"""Finishing the heads of a mixer (csrc/kernels/head_norm.cu): norm, weight and gate of a recurrence's raw outputs, and
the sigmoid gate of attention outputs."""
from __future__ import annotations

import torch

from . import _lib
from ._lib import F, I, L, P, check, ptr, stream

_lib.register_signature("xllm_head_norm_gate", [P, L, P, P, P, L, P, I, L, I, I, I, I, F, I, P])
_lib.register_signature("xllm_head_gate", [P, P, P, L, L, I, I, I, I, I, P])

_DT = {torch.bfloat16: 0, torch.float32: 1}
_ACT = {"silu": 0, "sigmoid": 1}


def head_norm_gate(o, out, div=None, g=None, w=None, unit_norm=True, act="silu", eps=1e-6):
    """out[t, h dv + i] = o[t, h, i] (/ div[t, h]) (/ rms over the head) (* w) (* act(g[t, h dv + i])).  o fp32 [T, H, dv];
    w [dv] is shared by the heads, [H * dv] has a value for each of their elements."""
    T, H, dv = o.shape
    per_head = w is not None and w.numel() == H * dv and H > 1
    if not o.is_cuda:
        x = o if div is None else o / torch.where(div > 0, div, torch.ones_like(div))[..., None]
        if unit_norm:
            x = x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)
        if w is not None:
            x = x * w.float().view(-1, dv)
        x = x.reshape(T, H * dv)
        if g is not None:
            x = x * (torch.nn.functional.silu(g.float()) if act == "silu" else torch.sigmoid(g.float()))
        out.copy_(x.to(out.dtype))
        return out
    assert o.dtype == torch.float32 and o.is_contiguous() and out.stride(1) == 1
    assert g is None or (g.stride(1) == 1 and g.dtype == out.dtype)
    check(_lib.load().xllm_head_norm_gate(ptr(out), out.stride(0), ptr(o), ptr(div), ptr(g), g.stride(0) if g is not None else 0,
                                          ptr(w), dv if per_head else 0, T, H, dv, int(unit_norm), _ACT[act], eps,
                                          _DT[out.dtype], stream()), "head_norm_gate")
    from . import _count
    _count()
    return out


def head_gate(a, g, dv):
    """a [T, H, d_pad] (heads of dv, stored wider) -> [T, H * dv] times sigmoid(g), g [T, H * dv] or one per head [T, H]."""
    T, H, dp = a.shape
    per_head = g.shape[1] == H and dv > 1
    if not a.is_cuda:
        if per_head:
            return (a[..., :dv].float() * torch.sigmoid(g.float())[..., None]).to(a.dtype).reshape(T, H * dv)
        return (a[..., :dv].reshape(T, H * dv).float() * torch.sigmoid(g.float())).to(a.dtype)
    assert a.is_contiguous() and g.stride(1) == 1 and g.dtype == a.dtype
    out = torch.empty((T, H * dv), dtype=a.dtype, device=a.device)
    check(_lib.load().xllm_head_gate(ptr(out), ptr(a), ptr(g), g.stride(0), T, H, dv, dp, int(per_head), _DT[a.dtype], stream()),
          "head_gate")
    from . import _count
    _count()
    return out
