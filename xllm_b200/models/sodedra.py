"""Sodedra: a small hybrid decoder of parallel layers.

Layers come in any order from the configuration: `mlstm` (matrix memory with exponential gates), `channel_delta` (gated
delta rule with a decay per key channel behind short convolutions) or `attention` (grouped queries over a sliding window
with an output gate), each with a dense SwiGLU feed-forward, a mixture of experts, or none.  Both sublayers of a layer read
one norm of the residual, which is fp32 throughout; norm weights are stored as their distance from one.

    h = norm1 x;   x <- x + mixer(h) + ff(h)

The mechanisms live in models/mixers.py and models/qwen_moe.py; this file reads the configuration and strings them together
so that a layer's residual update is one launch with the next layer's norm (ops/residual.py).  There is no counterpart in
the reference's zoo (xllm/models/llm/).
"""
from __future__ import annotations

import dataclasses
from types import SimpleNamespace

import torch

from ..ops.residual import residual_update
from ..parallel.state import single
from .layers import DenseMLP, LMHead, Module, RotaryEmbedding
from .mixers import DeltaRuleMixer, FusedProjection, MatrixMemoryMixer, WindowAttention, round_up
from .qwen_moe import SparseMoeBlock
from .registry import register_model
from .state import RecurrentStatePool


def _rope(rot, args, device):
    if int(rot["dims"]) == 0:
        return None
    s = rot.get("scaling")
    if s:
        s = {"rope_type": "llama3", "factor": s["factor"], "low_freq_factor": s["low"], "high_freq_factor": s["high"],
             "original_max_position_embeddings": s["original"]}
    return RotaryEmbedding(int(rot["dims"]), args.max_position_embeddings, float(rot["base"]), s or None, device)


class SodedraLayer(Module):
    def __init__(self, args, idx, dtype, device):
        super().__init__()
        spec, eps, W = args.extra["layers"][idx], args.rms_norm_eps, args.hidden_size
        m, self.idx = spec["mixer"], idx
        self.norm1 = self.add_param("norm1", torch.zeros(W, dtype=dtype, device=device))
        if spec["type"] == "mlstm":
            mixer = MatrixMemoryMixer(W, m["heads"], m["dim"], m["vdim"], m["gate_cap"], eps, dtype, device)
        elif spec["type"] == "channel_delta":
            mixer = DeltaRuleMixer(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], int(m["conv"]), int(m.get("a1", 16)),
                                   int(m.get("g1", 16)), eps, dtype, device)
        elif spec["type"] == "attention":
            mixer = WindowAttention(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["mask"]["size"], dtype,
                                    device, rope=_rope(m["rot"], args, device))
        else:
            raise ValueError(f"unknown mixer type {spec['type']!r} of layer {idx}")
        self.mixer = self.add_module("mix", mixer)
        self.proj = mixer.add_module("in", FusedProjection(W, mixer.width_parts(), dtype, device, biased=mixer.biased))
        small = [("mix." + n, w, b) for n, w, b in mixer.small_parts()]
        self.small_names = [n for n, _, _ in mixer.small_parts()]
        self.mlp, self.moe, self.ff_to = None, False, 1
        f = spec.get("mlp")
        if f is not None and f["kind"] == "dense":
            self.ff_to = 8
            self.mlp = self.add_module("mlp", DenseMLP(W, round_up(int(f["ff"]), 8), "silu", dtype, device))
        elif f is not None and f["kind"] == "moe":
            r = f["router"]
            groups = r.get("groups") or {"count": 1, "keep": 1}
            E, G, K = int(r["experts"]), int(groups["count"]), int(r["top"])
            if E % G or int(groups["keep"]) * (E // G) < K:
                raise ValueError(f"layer {idx}: {groups['keep']} of {G} groups of {E} experts do not hold {K}")
            self.moe = True
            # the tensor-core product with the activation in its epilogue takes widths in steps of 64
            self.ff_to = 64 if torch.device(device).type == "cuda" and dtype == torch.bfloat16 else 1
            a = dataclasses.replace(
                args, num_experts=E, num_experts_per_tok=K, moe_intermediate_size=round_up(int(f["expert"]["ff"]), self.ff_to),
                scoring_func="softmax", n_group=G, topk_group=int(groups["keep"]), norm_topk_prob=True, moe_group_score="max",
                routed_scaling_factor=float(r["scale"]), router_bias=True, n_shared_experts=0, fp8_execution=False)
            self.mlp = self.add_module("mlp", SparseMoeBlock(a, dtype, device, own_router=False))
            small.append(("mlp.router", E, False))
        elif f is not None:
            raise ValueError(f"unknown feed-forward kind {f['kind']!r} of layer {idx}")
        self.small = None
        if small:
            self.small = self.add_module("small", FusedProjection(W, [(n, w) for n, w, _ in small], dtype, device,
                                                                  biased=[n for n, _, b in small if b], f32=True))

    def forward(self, h, positions, meta, kv, state):
        """h: norm1 of the residual.  Returns the two branches (the second may be None)."""
        rows = self.proj(h)
        z = self.small(h) if self.small is not None else None
        small = {n: self.small.part(z, "mix." + n) for n in self.small_names}
        a = self.mixer(self.proj, rows, small, positions, meta, kv, state)
        if self.mlp is None:
            return a, None
        return a, self.mlp(h, logits=self.small.part(z, "mlp.router")) if self.moe else self.mlp(h)

    __call__ = forward


class SodedraCausalLM(Module):
    needs_state = True
    state_on_device = True          # state slots are a device input of the step: graphs capture it
    supports_graph = True
    supports_prefill_graph = True
    # the kernel sources a process that runs nothing but this model needs
    kernel_sources = ("gemm_tcgen05", "activation", "attn_decode", "attn_prefill", "attn_prefill_tc", "attn_generic",
                      "delta_rule", "mlstm", "head_norm", "proj_f32", "moe", "residual", "rope_norm_kv", "misc", "sampling")
    fused_tp = False

    def __init__(self, args, dtype=torch.bfloat16, device="cpu", ps=None):
        super().__init__()
        self.args, self.ps, self.dtype, self.device = args, ps or single(), dtype, torch.device(device)
        if self.ps.tp_size != 1:
            raise ValueError("Sodedra runs unsharded (one GPU per replica)")
        W = args.hidden_size
        self.embed = self.add_param("embed", torch.zeros(args.vocab_size, W, dtype=dtype, device=device))
        self.layers = [self.add_module(f"l{i}", SodedraLayer(args, i, dtype, device)) for i in range(args.num_hidden_layers)]
        self.final_norm = self.add_param("final.norm", torch.zeros(W, dtype=dtype, device=device))
        self.lm_head = LMHead(args.vocab_size, W, dtype, device, self.ps, tied=SimpleNamespace(weight=self.embed))
        self.state = None

    # ------------------------------------------------------------------ cache and state geometry
    def kv_layout(self):
        """Per layer: (planes, kv heads, head size) of its paged cache, or None."""
        return [l.mixer.kv_geometry() for l in self.layers]

    @property
    def num_kv_heads_local(self):
        return max([g[1] for g in self.kv_layout() if g] + [1])

    @property
    def head_dim(self):
        return max([g[2] for g in self.kv_layout() if g] + [64])

    def _state_shapes(self):
        return {l.idx: l.mixer.state_parts() for l in self.layers if l.mixer.state_parts() is not None}

    def state_bytes_per_slot(self):
        return RecurrentStatePool.bytes_per_slot(self._state_shapes())

    def alloc_state(self, slots):
        self.state = RecurrentStatePool(self._state_shapes(), slots, self.device)
        return self.state

    # ------------------------------------------------------------------ weights
    def remap_weight(self, name, w):
        base, _, leaf = name.rpartition(".")
        if leaf == "o" and base.endswith(".mix"):
            return [(name + ".weight", w)]
        if ".mlp" not in base or leaf == "router":
            return [(name, w)]
        if leaf == "correction":
            return [(base + ".gate.e_score_correction_bias", w)]
        # gate, up, down of the dense feed-forward or of expert e: its width rounded up with zeros
        dim = 1 if leaf == "down" else 0
        layer = self.layers[int(name[1:name.index(".")])]
        pad = round_up(w.shape[dim], layer.ff_to) - w.shape[dim]
        if pad:
            w = torch.nn.functional.pad(w, (0, pad) if dim == 1 else (0, 0, 0, pad))
        owner, _, expert = base.rpartition(".")
        if expert == "mlp":
            return [(f"{base}.{leaf}_proj.weight", w)]
        return [(f"{owner}.experts.{expert[1:]}.{leaf}_proj.weight", w)]

    def init_random(self, std=0.02, seed=0):
        super().init_random(std, seed)
        for name, t in self.named_params():
            if name.endswith("mix.norm"):
                t.fill_(1.0)
            elif name.endswith(".conv"):
                t[-1] += 1.0
            elif name.endswith("dt_bias"):
                t.fill_(-4.0)                               # decays near one
            elif name.endswith("small.bias"):
                t.fill_(2.0)                                # forget gates near one
            elif t.dim() == 1:
                t.zero_()

    # ------------------------------------------------------------------ forward
    def forward(self, tokens, positions, meta, kv_caches, embeds=None):
        """tokens, positions [T] int64 -> final-norm hidden states [T, width] in the model's dtype."""
        norm = dict(eps=self.args.rms_norm_eps, w_out_offset=1.0)
        norms = [l.norm1 for l in self.layers[1:]] + [self.final_norm]
        x, h = residual_update(None, self.embed, rows=tokens, coef=self.args.extra["embedding_scale"],
                               w_out=self.layers[0].norm1, **norm)
        for layer, kv, w_out in zip(self.layers, kv_caches, norms):
            a, b = layer(h, positions, meta, kv, self.state.layers.get(layer.idx))
            x, h = residual_update(x, a, y2=b, w_out=w_out, **norm)
        return h

    def logits(self, hidden_rows):
        return self.lm_head(hidden_rows)

    def logits_local(self, hidden_rows):
        return self.lm_head.forward_local(hidden_rows)

    def gather_logits(self, local):
        return self.lm_head.gather(local)

    def greedy_from_local(self, local):
        return self.lm_head.greedy_from_local(local)

    __call__ = forward


@register_model("sodedra", "Sodedra", kernel_sources=SodedraCausalLM.kernel_sources)
def build_sodedra(args, dtype, device, ps):
    return SodedraCausalLM(args, dtype, device, ps)
