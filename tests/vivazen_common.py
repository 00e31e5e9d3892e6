"""Configurations for the Vivazen tests."""
import copy

import torch

import vivazen_oracle as oracle
from femirax_common import LIMIT, row_errors


def rotation(dims, base=1000.0, factor=4.0, original=64, fast=8.0, slow=0.5):
    return {"base": base, "dims": dims, "scaling": {"factor": factor, "fast": fast, "original": original, "slow": slow}}


def attention(heads, kv, dim, vdim, conv, scale, softcap, ff=None):
    return {"type": "attention", "mlp": None if ff is None else {"ff": ff, "kind": "dense"},
            "mixer": {"conv": conv, "dim": dim, "heads": heads, "kv_heads": kv, "scale": scale, "softcap": softcap, "vdim": vdim}}


def latent(heads, dim, vdim, rank, rot, window, scale, ff=None):
    return {"type": "latent_attention", "mlp": None if ff is None else {"ff": ff, "kind": "dense"},
            "mixer": {"dim": dim, "heads": heads, "kv_rank": rank, "mask": {"size": window}, "rot": rot, "rot_dim": rot["dims"],
                      "scale": scale, "vdim": vdim}}


def again(layer, j):
    """The same layer with the tensors of layer j."""
    return dict(copy.deepcopy(layer), weights_of=j)


def config(layers, vocab=104, width=72, eps=1e-5, groups=2, alpha=1.7):
    return {"architecture": "Vivazen", "layers": layers, "norm": {"eps": eps, "groups": groups}, "postln_alpha": alpha, "vocab": vocab,
            "width": width}


_A = attention(6, 2, 20, 14, 3, 0.3, 12.0, ff=50)
_L = latent(5, 14, 22, 26, rotation(10), 21, 0.27, ff=36)
_BIG = latent(4, 64, 128, 512, rotation(64, base=1e4, original=512, fast=32.0, slow=1.0), 40, 0.1, ff=128)
CONFIGS = {
    # odd sizes everywhere: nothing a multiple of eight, lent tensors of both kinds, layers without a feed-forward
    "odd": config([_L, _A, again(_L, 0), latent(3, 9, 5, 7, rotation(2, base=20.0), 2, 0.5), again(_A, 1),
                   attention(4, 1, 10, 36, 2, 0.4, 30.0)], groups=3),
    # aligned sizes: tensor-core kernels at several widths, one norm part, no sum's factor
    "aligned": config([attention(16, 4, 128, 128, 4, 0.09, 50.0, ff=128), _BIG, again(_BIG, 1), attention(4, 4, 64, 64, 3, 0.125, 20.0),
                       latent(5, 40, 48, 80, rotation(32), 30, 0.2, ff=192)], vocab=128, width=128, eps=1e-6, groups=1, alpha=1.0),
    # rows of 256, heads wider than the values and the other way round, many parts, one tap, scaling that changes nothing
    "wide": config([latent(3, 80, 40, 160, rotation(48, factor=1.0), 75, 0.1, ff=64), attention(3, 3, 144, 24, 1, 0.1, 8.0),
                    attention(2, 1, 24, 200, 5, 0.3, 40.0, ff=72)], vocab=64, width=96, groups=12, alpha=3.0),
    # a width and a vocabulary that no tensor-core product takes
    "ragged": config([attention(3, 3, 22, 10, 3, 0.3, 9.0, ff=30), latent(2, 16, 70, 30, rotation(8), 16, 0.3)], vocab=101, width=100,
                     groups=5, alpha=0.8),
    # windows in every layer: pages behind them return, nothing recurs
    "windows": config([latent(4, 16, 16, 24, rotation(16), 34, 0.25, ff=40), latent(3, 20, 8, 40, rotation(6), 9, 0.3)], groups=4),
}


def weights_of(name, seed=0):
    return CONFIGS[name], oracle.random_weights(CONFIGS[name], seed)


def expect(cfg, weights, tokens):
    return oracle.forward(tokens, cfg, {n: t.double() for n, t in weights.items()})


def row_limits(cfg, weights, tokens, want, dtype):
    """Per place of one sequence: the error a correct implementation may show."""
    lim = torch.full((len(tokens),), LIMIT[dtype], dtype=torch.float64)
    if dtype == "bfloat16":
        for seed in range(12):
            oracle.NOISE = torch.Generator().manual_seed(seed)
            try:
                lim = torch.maximum(lim, 3 * row_errors(expect(cfg, weights, tokens), want))
            finally:
                oracle.NOISE = None
    return lim
