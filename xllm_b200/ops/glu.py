"""Gated activations of feed-forward layers: act(gate) * up by name ("silu", "gelu", "gelu_tanh"), or a ClampedGLU."""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as Fn

_CODES = {"silu": 0, "gelu": 1, "gelu_tanh": 2, "gelu_pytorch_tanh": 2}


@dataclass(frozen=True)
class ClampedGLU:
    """g sigmoid(alpha g) (u + 1) with g = min(gate, limit) and u = up clamped to +-limit."""
    limit: float
    alpha: float = 1.702

    def __post_init__(self):
        if not self.limit > 0:
            raise ValueError("a clamped activation needs a positive limit")


def code(act):
    """(code, limit, alpha) as the kernels take it; the epilogues of the GEMMs count from one."""
    return (3, float(act.limit), float(act.alpha)) if isinstance(act, ClampedGLU) else (_CODES[act], 0.0, 0.0)


def known(act):
    return isinstance(act, ClampedGLU) or act in _CODES


def apply(gate, up, act):
    """In the tensors' dtype (fp32 in, fp32 out)."""
    if isinstance(act, ClampedGLU):
        g = gate.clamp(max=act.limit)
        return g * torch.sigmoid(act.alpha * g) * (up.clamp(-act.limit, act.limit) + 1.0)
    if act == "silu":
        return Fn.silu(gate) * up
    return Fn.gelu(gate, approximate="none" if act == "gelu" else "tanh") * up
