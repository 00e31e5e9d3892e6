"""Configurations and limits for the Sodedra tests (engines, checkpoints and error measures are those of Femirax)."""
import torch

import sodedra_oracle as oracle
from femirax_common import LIMIT, row_errors


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale=1.0, groups=None):
    r = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def mlstm(heads, dim, vdim, cap=12.0, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def delta(heads, kv, dim, vdim, conv=4, mlp=None):
    return {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def attention(heads, kv, dim, vdim, window, rot, scale, base=2000.0, scaling=None, mlp=None):
    r = {"base": base, "dims": rot}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
                                                       "mask": {"size": window}, "rot": r}}


def config(layers, vocab=104, width=72, eps=1e-5, scale=2.0):
    return {"architecture": "Sodedra", "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": scale}, "vocab": vocab,
            "width": width}


CONFIGS = {
    # nothing a multiple of eight, shared query/key heads, unequal layers and windows, values wider and narrower than keys
    "odd": (config([delta(6, 2, 20, 14, conv=3, mlp=moe(6, 2, 20, 1.7, (3, 2))),
                    attention(6, 2, 20, 12, 21, 12, 0.31, scaling=(3.0, 1.0, 3.0, 40), mlp=dense(50)),
                    mlstm(3, 26, 10, cap=5.0, mlp=moe(10, 3, 28, 0.6, (5, 3))),
                    delta(1, 1, 10, 30, conv=2),
                    attention(5, 1, 10, 36, 34, 10, 0.2, mlp=moe(5, 1, 12))]), (5, 9)),
    # aligned sizes: the tensor-core kernels at head sizes 64 and 128, experts in the grouped product
    "aligned": (config([mlstm(2, 64, 32, mlp=dense(96)),
                        attention(4, 2, 128, 128, 40, 64, 0.09, scaling=(8.0, 1.0, 4.0, 64), mlp=moe(16, 4, 64, 2.5, (8, 5))),
                        delta(4, 2, 32, 64, mlp=dense(64)),
                        attention(4, 4, 64, 32, 16, 16, 0.125, mlp=moe(8, 2, 40, 1.0, (2, 1)))], vocab=128, width=128,
                       eps=1e-6, scale=1.0), (24, 16)),
    # large heads; no attention first, no feed-forward on some
    "wide": (config([delta(2, 1, 200, 72, conv=5), mlstm(1, 144, 160, cap=20.0),
                     attention(2, 2, 144, 200, 50, 8, 0.09, mlp=dense(40))], vocab=64, width=96), (16, 8)),
    # a width and a vocabulary that no tensor-core product takes
    "ragged": (config([attention(3, 3, 22, 22, 9, 0, 0.2, mlp=moe(4, 2, 10)), delta(2, 2, 6, 70, conv=1, mlp=dense(30)),
                       mlstm(2, 10, 34)], vocab=101, width=100, scale=0.7), (7, 3)),
    "recurrent_only": (config([mlstm(2, 16, 16, mlp=dense(24)), delta(2, 2, 16, 24, mlp=moe(4, 2, 16, 1.0, (2, 2)))]), (4, 4)),
}


def weights_of(name, seed=0):
    cfg, rank = CONFIGS[name]
    return cfg, oracle.random_weights(cfg, rank, seed)


def expect(cfg, weights, tokens):
    return oracle.forward(tokens, cfg, {n: t.double() for n, t in weights.items()})


def row_limits(cfg, weights, tokens, want, dtype):
    """Per place of one sequence: the error a correct implementation may show."""
    lim = torch.full((len(tokens),), LIMIT[dtype], dtype=torch.float64)
    if dtype == "bfloat16":
        for seed in range(16):
            oracle.NOISE = torch.Generator().manual_seed(seed)
            try:
                lim = torch.maximum(lim, 3 * row_errors(expect(cfg, weights, tokens), want))
            finally:
                oracle.NOISE = None
    return lim
