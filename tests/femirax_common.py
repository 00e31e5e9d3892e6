"""Configurations, checkpoints and engines for the Femirax tests."""
import json
import os

import pytest
import torch

import femirax_oracle as oracle
from xllm_b200.engine.llm_engine import EngineConfig, LLMEngine
from xllm_b200.utils.loader import save_file

TARGETS = [pytest.param(("cpu", "float32"), id="cpu-fp32"),
           pytest.param(("cuda:0", "float32"), id="gpu-fp32", marks=pytest.mark.gpu),
           pytest.param(("cuda:0", "bfloat16"), id="gpu-bf16", marks=pytest.mark.gpu)]
# root mean square of a row's error over that of the logits; in bfloat16 a row may be off by more where rounding alone
# (the plain implementation with jittered activations) moves it by more
LIMIT = {"float32": 2e-4, "bfloat16": 0.06}


def retention(heads, dim, vdim, decay, rot, base=500.0, ff=None):
    return {"type": "retention", "mlp": None if ff is None else {"ff": ff, "kind": "dense"},
            "mixer": {"decay": decay, "dim": dim, "heads": heads, "rot": {"base": base, "dims": rot}, "vdim": vdim}}


def parallel(heads, kv, dim, rot, scale, rheads, rdim, rvdim, tau, base=2000.0, ff=None):
    return {"type": "parallel", "mlp": None if ff is None else {"ff": ff, "kind": "dense"},
            "mixer": {"left": {"dim": dim, "heads": heads, "kv_heads": kv, "rot": {"base": base, "dims": rot},
                               "scale": scale, "vdim": dim},
                      "right": {"dim": rdim, "heads": rheads, "tau": tau, "vdim": rvdim}}}


def config(layers, vocab=104, width=72, eps=1e-5, side=6):
    return {"architecture": "Femirax", "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side},
            "vocab": vocab, "width": width}


CONFIGS = {
    # odd sizes everywhere: nothing a multiple of eight, partial rotations, one key/value head, unequal layers
    "odd": (config([parallel(6, 2, 20, 12, 0.31, 3, 10, 14, 4.0, ff=50),
                    retention(2, 26, 38, [0.9, 0.997], 18),
                    retention(3, 12, 6, [0.5, 0.98, 1.0], 12, ff=44),
                    parallel(5, 1, 36, 36, 0.2, 1, 18, 9, 1.0)]), 5),
    # aligned sizes: the tensor-core kernels at head sizes 64 and 128, a side input wider than a vector
    "aligned": (config([retention(4, 32, 64, [0.95, 0.99, 0.999, 0.9999], 32, ff=96),
                        parallel(4, 4, 64, 32, 0.125, 2, 64, 32, 16.0),
                        parallel(4, 1, 128, 128, 0.05, 2, 128, 96, 8.0, ff=128),
                        retention(1, 128, 160, [0.98], 64)], vocab=128, width=128, side=24, eps=1e-6), 24),
    # large heads, no feed-forward anywhere, no parallel layer first
    "wide": (config([retention(2, 200, 72, [0.97, 0.9995], 40),
                     parallel(2, 2, 144, 8, 0.09, 1, 192, 80, 2.0)], vocab=64, width=96, side=8), 16),
    # a width and a vocabulary that no tensor-core product takes
    "ragged": (config([parallel(3, 3, 22, 8, 0.2, 2, 34, 26, 3.0, ff=30), retention(2, 10, 70, [0.96, 0.8], 6)],
                      vocab=101, width=100, side=5), 7),
    "retention_only": (config([retention(2, 16, 16, [0.9, 0.99], 8, ff=24), retention(1, 40, 24, [0.95], 40)], side=3), 4),
}


def weights_of(name, seed=0):
    cfg, rank = CONFIGS[name]
    return cfg, oracle.random_weights(cfg, rank, seed)


def write_checkpoint(path, cfg, weights):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(weights, os.path.join(path, "model.safetensors"))
    return str(path)


def make_engine(path, cfg, weights, target, **kw):
    device, dtype = target
    opt = dict(block_size=16, num_blocks=64, max_seqs_per_batch=4, max_running_seqs=4, max_tokens_per_batch=1024,
               max_model_len=1024, max_sample_rows=1024)
    opt.update(kw)
    return LLMEngine(EngineConfig(model=write_checkpoint(path, cfg, weights), dtype=dtype, device=device, **opt))


def expect(cfg, weights, tokens):
    return oracle.forward(tokens, cfg, {n: t.double() for n, t in weights.items()})


def random_tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def row_errors(got, want):
    """rms of every row's difference (mean taken off) over the rms of all wanted logits."""
    d = got.double() - want.double()
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / scale


def error(got, want):
    return float(row_errors(got, want).max())


def row_limits(cfg, weights, tokens, want, dtype):
    """Per place of one sequence: the error a correct implementation may show."""
    lim = torch.full((len(tokens),), LIMIT[dtype], dtype=torch.float64)
    if dtype == "bfloat16":
        for seed in range(24):
            oracle.NOISE = torch.Generator().manual_seed(seed)
            try:
                lim = torch.maximum(lim, 3 * row_errors(expect(cfg, weights, tokens), want))
            finally:
                oracle.NOISE = None
    return lim


def close(got, want, limits):
    """All rows within one and a half times their limit and at most a fiftieth (or one) above it."""
    r = row_errors(got, want) / limits
    return bool(r.max() <= 1.5 and int((r > 1).sum()) <= max(1, len(r) // 50)), float(r.max())


def feed(engine, rid, tokens, cuts, end=True):
    """One request alone, cut into portions of the sizes `cuts` (repeated); logits of every place."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(cuts[i % len(cuts)], len(tokens) - at)
        out.append(engine.replay_step([(rid, tokens[at:at + n], list(range(n)))]))
        at, i = at + n, i + 1
    if end:
        engine.replay_end(rid)
    return torch.cat(out)
