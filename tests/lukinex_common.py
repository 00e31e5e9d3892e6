"""Configurations and limits for the Lukinex tests (engines, checkpoints and error measures are those of Femirax)."""
import torch

import lukinex_oracle as oracle
from femirax_common import LIMIT, row_errors


def moe(experts, top, ff, limit, shared_ff, shared_limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top},
            "shared": {"ff": shared_ff, "limit": shared_limit}}


def rotation(dims, base=2000.0, factor=None):
    r = {"base": base, "dims": dims}
    if factor is not None:
        r["scaling"] = {"factor": factor}
    return r


def mask(size, keep):
    return {"size": size, "keep_first": keep}


def attention(heads, kv, dim, vdim, seen, rot, scale, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim,
                                                       "mask": mask(*seen), "rot": rot, "scale": scale}}


def parallel(heads, kv, dim, vdim, seen, rot, scale, conv, softcap, rheads, rdim, rvdim, decay, mlp=None):
    return {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "mask": mask(*seen), "rot": rot, "scale": scale,
                 "conv": conv, "softcap": softcap},
        "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": decay}}}


def latent(heads, dim, vdim, q_rank, kv_rank, scale, source=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale}
    if source is not None:
        m["kv_from"] = source
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def config(layers, vocab=104, width=72, eps=1e-5):
    return {"architecture": "Lukinex", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # nothing a multiple of eight, values wider and narrower than keys, latents used twice with other heads
    "odd": config([latent(3, 12, 10, 18, 26, 0.4, mlp=moe(5, 2, 20, 0.9, 12, 1.3)),
                   parallel(6, 2, 20, 14, (21, 5), rotation(12), 0.31, 3, 5.0, 3, 10, 18, [0.5, 0.95, 0.9995],
                            mlp=moe(7, 3, 28, 1.1, 20, 0.7)),
                   attention(5, 1, 10, 36, (34, 1), rotation(6, factor=3.0), 0.5),
                   latent(2, 20, 22, 14, 26, 0.3, source=0),
                   parallel(2, 2, 26, 38, (9, 18), rotation(26), 0.2, 2, 2.0, 1, 22, 6, [0.97])]),
    # aligned sizes: the tensor-core kernels at head sizes 64 and 128, latent rows of 128, grouped experts
    "aligned": config([parallel(4, 2, 128, 128, (40, 20), rotation(64), 0.09, 4, 8.0, 2, 64, 32, [0.9, 0.999],
                                mlp=moe(16, 4, 64, 1.2, 64, 0.8)),
                       latent(4, 128, 128, 64, 128, 0.09, mlp=moe(8, 2, 40, 1.0, 24, 1.0)),
                       attention(4, 4, 64, 32, (16, 16), rotation(16, factor=2.0), 0.125, mlp=moe(4, 1, 64, 0.5, 128, 2.0)),
                       latent(2, 64, 64, 32, 128, 0.125, source=1),
                       parallel(4, 4, 64, 64, (33, 0), rotation(64, base=1e5), 0.125, 3, 20.0, 4, 32, 64,
                                [0.7, 0.9, 0.99, 1.0])], vocab=128, width=128, eps=1e-6),
    # latent rows of 512 and 256 under more heads than a tile, large heads, more taps than the vector kernel takes
    "wide": config([latent(20, 24, 32, 40, 300, 0.25), latent(3, 128, 128, 48, 200, 0.1, mlp=moe(6, 2, 24, 1.0, 40, 1.0)),
                    parallel(2, 1, 144, 200, (50, 7), rotation(8), 0.09, 6, 12.0, 1, 200, 72, [0.98]),
                    latent(17, 16, 8, 16, 300, 0.3, source=0)], vocab=64, width=96),
    # a width and a vocabulary that no tensor-core product takes, one expert of four, no rotation, convolution of one tap
    "ragged": config([parallel(3, 3, 22, 22, (11, 2), rotation(0), 0.2, 1, 3.0, 2, 6, 70, [0.9, 0.96], mlp=moe(4, 1, 10, 0.8, 30, 1.5)),
                      latent(2, 10, 34, 9, 15, 0.3), attention(3, 1, 14, 14, (13, 4), rotation(14), 0.3)], vocab=101, width=100),
    # latents beyond the rows of the tensor-core kernels, heads beyond theirs, a decay of nothing
    "beyond": config([latent(3, 40, 24, 30, 600, 0.2), attention(2, 1, 320, 264, (19, 3), rotation(64), 0.06),
                      parallel(2, 2, 16, 16, (12, 12), rotation(16), 0.25, 3, 4.0, 2, 264, 136, [0.0, 0.99])]),
    # only windows: pages between the kept tokens and the window return
    "windows": config([attention(4, 2, 16, 16, (30, 18), rotation(16), 0.25, mlp=moe(4, 2, 16, 1.0, 16, 1.0)),
                       parallel(2, 2, 16, 24, (34, 5), rotation(8), 0.25, 3, 6.0, 2, 16, 24, [0.9, 0.99])]),
    # no state beside the cache
    "stateless": config([latent(2, 16, 16, 16, 24, 0.25), attention(2, 1, 16, 16, (20, 3), rotation(16), 0.25),
                         latent(2, 16, 16, 16, 24, 0.25, source=0, mlp=moe(3, 2, 16, 1.0, 16, 1.0))]),
}


def clear_routing(cfg, w, dims=8, gap=0.15, seed=0):
    """Routers that read `dims` coordinates which only the embedding writes, and embeddings whose routing is no close call in
    any layer: rounding must not decide which experts a token visits."""
    g = torch.Generator().manual_seed(seed)
    readers = []
    for i, layer in enumerate(cfg["layers"]):
        for n in ("norm1b", "norm2b"):
            if f"l{i}.{n}" in w:
                w[f"l{i}.{n}"][:dims] = 0.0
        if layer["mlp"] is not None:
            r = w[f"l{i}.mlp.router"]
            r[:] = 0.0
            r[:, :dims] = (torch.randn(r.shape[0], dims, generator=g) * 2.0).to(r.dtype)
            readers.append((r[:, :dims].float() * w[f"l{i}.norm2"][:dims].float(), layer["mlp"]["router"]["top"]))
    for t in range(cfg["vocab"]):
        while True:
            code = torch.randn(dims, generator=g).to(torch.bfloat16)
            zs = [(r @ code.float()).sort(descending=True).values for r, _ in readers]
            if all(k == len(z) or float(z[k - 1] - z[k]) > gap * float(z.std()) for z, (_, k) in zip(zs, readers)):
                break
        w["embed"][t, :dims] = code
    return w


def weights_of(name, seed=0):
    return CONFIGS[name], clear_routing(CONFIGS[name], oracle.random_weights(CONFIGS[name], seed))


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
