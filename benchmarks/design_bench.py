#!/usr/bin/env python
"""Prefill and decode throughput of one model design beside the framework's closest models (Qwen3-Next: three
gated-delta-net layers per attention layer; others where a design has more in common with them) at equal size, random
weights, one GPU.

    python bench.py --design femirax [--steps K] [--warmup W]      # prints one JSON line
    python bench.py --design sodedra
    python bench.py --design lukinex
    python bench.py --design vivazen

Prefill: four prompts of 2048 tokens in one step.  Decode: 64 sequences of 512 prompt tokens, one token each per step.
Both go through the engine (scheduler, state slots, cache, sampling) and are timed with CUDA events around K steps
after W untimed ones; the weights and states of every size are larger than L2.
"""
from __future__ import annotations

import json
import os
import sys

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))

SIZES = {"1024": 1024, "2048": 2048, "4096": 4096}
LAYERS, VOCAB, SIDE = 8, 32768, 64
EXPERTS, TOP = 32, 4


def femirax_args(W):
    from xllm_b200.models import model_args_from_dict
    H = W // 128
    decay = [1.0 - 2.0 ** (-5 - 5 * h / max(H - 1, 1)) for h in range(H)]
    mlp = {"ff": 3 * W, "kind": "dense"}
    ret = {"type": "retention", "mlp": mlp, "mixer": {"heads": H, "dim": 128, "vdim": 128, "decay": decay,
                                                      "rot": {"base": 1e6, "dims": 128}}}
    par = {"type": "parallel", "mlp": mlp, "mixer": {
        "left": {"heads": H, "kv_heads": max(1, H // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                 "rot": {"base": 1e6, "dims": 128}},
        "right": {"heads": H, "dim": 128, "vdim": 128, "tau": 16.0, "rank": 16}}}
    return model_args_from_dict({"architecture": "Femirax", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6},
                                 "token_side": {"dim": SIDE}, "layers": [par if i % 4 == 3 else ret for i in range(LAYERS)]})


def sodedra_args(W):
    """Two delta-rule layers and one matrix-memory layer per attention layer; every other layer with experts."""
    from xllm_b200.models import model_args_from_dict
    H = W // 128
    dense = {"ff": 3 * W, "kind": "dense"}
    moe = {"kind": "moe", "expert": {"ff": W // 2},
           "router": {"experts": EXPERTS, "top": TOP, "scale": 1.0, "groups": {"count": 8, "keep": 4}}}
    delta = ("channel_delta", {"heads": H, "kv_heads": H, "dim": 128, "vdim": 128, "conv": 4, "a1": 128, "g1": 128})
    mlstm = ("mlstm", {"heads": H, "dim": 128, "vdim": 128, "gate_cap": 15.0})
    att = ("attention", {"heads": H, "kv_heads": max(1, H // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                         "mask": {"size": 1024}, "rot": {"base": 1e6, "dims": 128}})
    kinds = [delta, mlstm, delta, att]
    layers = [{"type": kinds[i % 4][0], "mixer": dict(kinds[i % 4][1]), "mlp": moe if i % 2 else dense} for i in range(LAYERS)]
    return model_args_from_dict({"architecture": "Sodedra", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6},
                                 "embedding": {"scale": 1.0}, "layers": layers})


def lukinex_args(W):
    """Two parallel layers, one normed attention layer and one latent attention layer in turn, of which the second latent layer
    reads the first one's latents; every layer with experts and a shared one."""
    from xllm_b200.models import model_args_from_dict
    H = W // 128
    heads = {"heads": H, "kv_heads": max(1, H // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
             "mask": {"size": 1024, "keep_first": 16}, "rot": {"base": 1e6, "dims": 128}}
    par = ("parallel", {"left": {**heads, "conv": 4, "softcap": 30.0},
                        "right": {"heads": H, "dim": 128, "vdim": 128,
                                  "decay": [1.0 - 2.0 ** (-5 - 5 * h / max(H - 1, 1)) for h in range(H)]}})
    att = ("attention", {**heads, "rot": {"base": 1e6, "dims": 64, "scaling": {"factor": 4.0}}})
    lat = ("latent_attention", {"heads": H, "dim": 128, "vdim": 128, "q_rank": W // 2, "kv_rank": 512, "scale": 128 ** -0.5})
    kinds = [par, lat, par, att]
    moe = {"kind": "moe", "expert": {"ff": W // 2, "limit": 7.0}, "router": {"experts": EXPERTS, "top": TOP},
           "shared": {"ff": W // 2, "limit": 7.0}}
    layers = [{"type": kinds[i % 4][0], "mixer": dict(kinds[i % 4][1]), "mlp": moe} for i in range(LAYERS)]
    layers[5]["mixer"]["kv_from"] = 1
    return model_args_from_dict({"architecture": "Lukinex", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6}, "layers": layers})


def vivazen_args(W):
    """Mixed-head attention and rotated latent attention in turn; the second latent layer uses the first one's tensors."""
    from xllm_b200.models import model_args_from_dict
    H = W // 128
    att = ("attention", {"heads": H, "kv_heads": max(1, H // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "conv": 4, "softcap": 30.0})
    lat = ("latent_attention", {"heads": H, "dim": 64, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 128 ** -0.5,
                                "mask": {"size": 1024}, "rot": {"base": 1e6, "dims": 64, "scaling": {
                                    "factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}})
    kinds = [att, lat]
    layers = [{"type": kinds[i % 2][0], "mixer": dict(kinds[i % 2][1]), "mlp": {"kind": "dense", "ff": 3 * W}} for i in range(LAYERS)]
    layers[3]["weights_of"] = 1
    return model_args_from_dict({"architecture": "Vivazen", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6, "groups": 4},
                                 "postln_alpha": 2.0, "layers": layers})


def lukinex_dense_args(W):
    """Windowed attention and latent attention in turn; one expert and a shared one, together as wide as a dense feed-forward."""
    from xllm_b200.models import model_args_from_dict
    a, layers = lukinex_args(W), []
    moe = {"kind": "moe", "expert": {"ff": 3 * W // 2, "limit": 7.0}, "router": {"experts": 1, "top": 1},
           "shared": {"ff": 3 * W // 2, "limit": 7.0}}
    att = {**next(l["mixer"] for l in a.extra["layers"] if l["type"] == "attention")}
    lat = {**next(l["mixer"] for l in a.extra["layers"] if l["type"] == "latent_attention"), "q_rank": W}
    for i in range(LAYERS):
        layers.append({"type": ("attention", "latent_attention")[i % 2], "mixer": dict((att, lat)[i % 2]), "mlp": moe})
    return model_args_from_dict({"architecture": "Lukinex", "vocab": VOCAB, "width": W, "norm": {"eps": 1e-6}, "layers": layers})


def qwen3_next_args(W):
    from xllm_b200.models import ModelArgs
    H = W // 128
    return ModelArgs(model_type="qwen3_next", vocab_size=VOCAB, hidden_size=W, num_hidden_layers=LAYERS, num_attention_heads=H,
                     num_key_value_heads=max(1, H // 4), head_dim=128, intermediate_size=3 * W, qk_norm=True, rope_theta=1e6,
                     max_position_embeddings=32768, tie_word_embeddings=False,
                     extra=dict(linear_num_value_heads=H, linear_num_key_heads=H, linear_key_head_dim=128,
                                linear_value_head_dim=128, linear_conv_kernel_dim=4, full_attention_interval=4))


def qwen3_next_moe_args(W):
    import dataclasses
    return dataclasses.replace(qwen3_next_args(W), num_experts=EXPERTS, num_experts_per_tok=TOP, moe_intermediate_size=W // 2,
                               moe_layer_freq=2)


def sodedra_moe_args(W):
    """Every layer with experts (Sodedra has no shared one: one more of them is used)."""
    a = sodedra_args(W)
    moe = next(l["mlp"] for l in a.extra["layers"] if l["mlp"]["kind"] == "moe")
    for l in a.extra["layers"]:
        l["mlp"] = {**moe, "router": {**moe["router"], "top": TOP + 1, "groups": {"count": 8, "keep": 5}}}
    return a


def qwen3_next_shared_args(W):
    """Every layer with the same experts and a shared one."""
    import dataclasses
    return dataclasses.replace(qwen3_next_moe_args(W), moe_layer_freq=1, n_shared_experts=1, shared_expert_intermediate_size=W // 2)


# name -> (title, arguments of the design, {model beside it: its arguments})
DESIGNS = {"femirax": ("Femirax", femirax_args, {"qwen3_next": qwen3_next_args}),
           "sodedra": ("Sodedra", sodedra_args, {"qwen3_next": qwen3_next_moe_args}),
           "lukinex": ("Lukinex", lukinex_args, {"qwen3_next": qwen3_next_shared_args, "sodedra": sodedra_moe_args}),
           "vivazen": ("Vivazen", vivazen_args, {"qwen3_next": qwen3_next_args, "lukinex": lukinex_dense_args})}


def engine_of(args):
    from xllm_b200.engine.llm_engine import EngineConfig, LLMEngine
    return LLMEngine(EngineConfig(model="bench", device="cuda:0", dtype="bfloat16", block_size=16, num_blocks=64 * 48 + 1,
                                  max_seqs_per_batch=64, max_tokens_per_batch=8192, max_model_len=2304, random_weights=True,
                                  enable_prefix_cache=False), model_args=args)


def timed(fn, n):
    import torch
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(n):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / n


def measure(args, steps, warmup):
    """{"prefill_tok_s", "decode_tok_s", ...} of one model."""
    import torch
    from xllm_b200 import ops
    eng = engine_of(args)
    g = torch.Generator().manual_seed(0)
    prompts = torch.randint(0, VOCAB, (4, 2048), generator=g).tolist()
    count = [0]
    base = ops.launches() + eng.runner.graph_launches

    def prefill():
        for p in prompts:
            count[0] += 1
            eng.add_request(f"p{count[0]}", p, max_tokens=1, temperature=0.0, ignore_eos=True)
        while eng.has_unfinished():
            eng.step()

    for _ in range(max(2, warmup // 2)):
        prefill()
    ms_p = timed(prefill, max(2, steps // 8))
    short = torch.randint(0, VOCAB, (64, 512), generator=g).tolist()
    for i, p in enumerate(short):
        eng.add_request(f"d{i}", p, max_tokens=1500, temperature=0.0, ignore_eos=True)
    while eng.scheduler.num_waiting or eng.scheduler.num_prefilling:
        eng.step()
    for _ in range(warmup):
        eng.step()
    ms_d = timed(eng.step, steps)
    for i in range(64):
        eng.abort(f"d{i}")
    out = {"prefill_tok_s": round(8192 / ms_p * 1e3), "prefill_ms": round(ms_p, 3), "decode_tok_s": round(64 / ms_d * 1e3),
           "decode_ms": round(ms_d, 3), "cuda_graphs": bool(eng.runner.graphs),
           "launches": ops.launches() + eng.runner.graph_launches - base, "weights_mb": eng.model.param_bytes() >> 20}
    del eng
    torch.cuda.empty_cache()
    return out


def run(design, steps=40, warmup=8, sampler=None):
    title, make_args, beside = DESIGNS[design]
    rows = []
    launches = 0
    if sampler is not None:
        sampler.start()
    for name, W in SIZES.items():
        row = {"width": W}
        for model, make in ((design, make_args), *beside.items()):
            row[model] = measure(make(W), steps, max(3, warmup))
        launches += row[design]["launches"]
        for model in beside:
            for what in ("prefill", "decode"):
                row[f"{what}_ratio" + ("" if model == "qwen3_next" else f"_{model}")] = \
                    round(row[design][f"{what}_tok_s"] / row[model][f"{what}_tok_s"], 2)
        rows.append(row)
    clocks = sampler.stop() if sampler is not None else None
    big = rows[-1][design]
    print(json.dumps({
        "metric": f"{title} decode tok/s", "value": big["decode_tok_s"], "unit": "tok/s", "n_gpus": 1, "steps": steps,
        "warmup": warmup, "ms_per_step": big["decode_ms"], "higher_is_better": True, "scaling": "strong", "vs_baseline": None,
        "dtype": "bf16", "data": "synthetic tokens, random weights", "impl": "xllm_b200",
        "config": {"model": f"{title}, {LAYERS} layers, widths {list(SIZES.values())}, beside {', '.join(beside)} of equal size",
                   "prefill": "4 x 2048 tokens in one step", "decode": "64 sequences behind 512 prompt tokens",
                   "l2": "weights and states larger than L2"},
        "sizes": rows, "gpu_launches": launches, "clocks": clocks}), flush=True)


if __name__ == "__main__":
    run(sys.argv[1])
