"""Femirax: a small hybrid decoder.

Layers come in any order from the configuration: `retention` (linear attention with one decay constant per head) or
`parallel` (attention whose values are its keys, beside gated linear attention with a decay per key channel; both
outputs are normalised over the width and averaged), each with or without a dense SwiGLU feed-forward.  After a
layer's sublayers a per-token side input joins the residual, which is fp32 throughout.

    x <- x + mixer(norm1 x);   x <- x + ff(norm2 x);   x <- x + rms(proj(gelu(gate x) * side[token, layer])) * w

The mechanisms live in models/mixers.py; this file reads the configuration and strings them together so that every
residual update is one launch with the norm that follows it (ops/residual.py).  There is no counterpart in the
reference's zoo (xllm/models/llm/).
"""
from __future__ import annotations

import torch

from ..ops.residual import residual_update
from ..parallel.state import single
from .layers import DenseMLP, LMHead, Module, RotaryEmbedding
from .mixers import FusedProjection, KeyValueAttention, LinearAttentionMixer, TokenSideInput, round_up
from .registry import register_model
from .state import RecurrentStatePool


class FemiraxLayer(Module):
    def __init__(self, args, idx, dtype, device):
        super().__init__()
        spec, eps, W = args.extra["layers"][idx], args.rms_norm_eps, args.hidden_size
        m = spec["mixer"]
        self.idx, self.kind, self.eps = idx, spec["type"], eps
        one = lambda: torch.ones(W, dtype=dtype, device=device)

        def rope(r, interleaved):
            if int(r["dims"]) == 0:
                return None
            return RotaryEmbedding(int(r["dims"]), args.max_position_embeddings, float(r["base"]), None, device, interleaved)

        self.norm1 = self.add_param("norm1", one())
        self.left = None
        if self.kind == "retention":
            mix = self.linear = self.add_module("mix", LinearAttentionMixer(
                W, m["heads"], m["dim"], m["vdim"], eps, dtype, device, decay=m["decay"], k_scale=m["dim"] ** -0.5,
                rope=rope(m["rot"], False)))
            parts = self.linear.width_parts()
        elif self.kind == "parallel":
            mix, l, r = self.add_module("mix", Module()), m["left"], m["right"]
            if int(l.get("vdim", l["dim"])) != int(l["dim"]):
                raise ValueError("parallel: the left mixer's values are its keys, so vdim must equal dim")
            self.left = mix.add_module("left", KeyValueAttention(W, l["heads"], l["kv_heads"], l["dim"], l["scale"], eps, dtype,
                                                                 device, rope=rope(l["rot"], True), prefix="left."))
            self.linear = mix.add_module("right", LinearAttentionMixer(
                W, r["heads"], r["dim"], r["vdim"], eps, dtype, device, rank=int(r.get("rank", 16)), tau=r["tau"],
                q_scale=r["dim"] ** -0.5, norm_weight=True, prefix="right."))
            self.left_out = mix.add_param("left.out", one())
            self.right_out = mix.add_param("right.out", one())
            parts = self.left.width_parts() + self.linear.width_parts()
        else:
            raise ValueError(f"unknown mixer type {self.kind!r} of layer {idx}")
        self.proj = mix.add_module("in", FusedProjection(W, parts, dtype, device))
        self.mlp = None
        if spec.get("mlp") is not None:
            if spec["mlp"].get("kind", "dense") != "dense":
                raise ValueError(f"unknown feed-forward kind {spec['mlp']['kind']!r} of layer {idx}")
            self.norm2 = self.add_param("norm2", one())
            self.mlp = self.add_module("mlp", DenseMLP(W, round_up(int(spec["mlp"]["ff"]), 8), "silu", dtype, device))
        dim = int(args.extra["side_dim"])
        self.side = self.add_module("side", TokenSideInput(W, dim, idx * dim, dtype, device))

    def forward(self, x, h, tokens, table, positions, meta, kv, state):
        """x: fp32 residual (updated in place); h: norm1(x).  Returns the side branch, which the next residual update
        normalises and adds."""
        rows = self.proj(h)
        y = self.linear(self.proj, rows, positions, meta, state)
        w_out = self.norm2 if self.mlp is not None else None
        if self.left is not None:
            a = self.left(self.proj, rows, positions, meta, *kv)
            _, h = residual_update(x, a, w=self.left_out, y2=y, w2=self.right_out, coef=0.5, w_out=w_out, eps=self.eps)
        else:
            _, h = residual_update(x, y, w_out=w_out, eps=self.eps)
        if self.mlp is not None:
            _, h = residual_update(x, self.mlp(h), eps=self.eps)
        return self.side(h, table, tokens)

    __call__ = forward


class FemiraxCausalLM(Module):
    needs_state = True
    state_on_device = True          # state slots are a device input of the step: graphs capture it
    supports_graph = True
    supports_prefill_graph = True
    # the kernel sources a process that runs nothing but this model needs
    kernel_sources = ("gemm_tcgen05", "activation", "attn_decode", "attn_prefill", "attn_prefill_tc", "attn_generic",
                      "linear_attn", "head_norm", "residual", "rope_norm_kv", "misc", "sampling")
    fused_tp = False

    def __init__(self, args, dtype=torch.bfloat16, device="cpu", ps=None):
        super().__init__()
        self.args, self.ps, self.dtype, self.device = args, ps or single(), dtype, torch.device(device)
        if self.ps.tp_size != 1:
            raise ValueError("Femirax runs unsharded (one GPU per replica)")
        W, n = args.hidden_size, args.num_hidden_layers
        self.embed = self.add_param("embed", torch.zeros(args.vocab_size, W, dtype=dtype, device=device))
        self.side_table = self.add_param("side.embed", torch.zeros(args.vocab_size, n * int(args.extra["side_dim"]), dtype=dtype,
                                                                   device=device))
        self.layers = [self.add_module(f"l{i}", FemiraxLayer(args, i, dtype, device)) for i in range(n)]
        self.final_norm = self.add_param("final.norm", torch.ones(W, dtype=dtype, device=device))
        self.lm_head = self.add_module("head", LMHead(args.vocab_size, W, dtype, device, self.ps))
        self.state = None

    # ------------------------------------------------------------------ cache and state geometry
    def kv_layout(self):
        """Per layer: (planes, kv heads, head size) of its paged cache, or None."""
        return [l.left.kv_geometry() if l.left is not None else None for l in self.layers]

    @property
    def num_kv_heads_local(self):
        return max([g[1] for g in self.kv_layout() if g] + [1])

    @property
    def head_dim(self):
        return max([g[2] for g in self.kv_layout() if g] + [64])

    def _state_shapes(self):
        return {l.idx: l.linear.state_shape for l in self.layers}

    def state_bytes_per_slot(self):
        return RecurrentStatePool.bytes_per_slot(self._state_shapes())

    def alloc_state(self, slots):
        self.state = RecurrentStatePool(self._state_shapes(), slots, self.device)
        return self.state

    # ------------------------------------------------------------------ weights
    def remap_weight(self, name, w):
        if name == "head":
            return [("head.weight", w)]
        base, _, leaf = name.rpartition(".")
        if leaf == "o" and ".mix" in base:
            return [(name + ".weight", w)]
        if base.endswith(".mlp") and leaf in ("gate", "up", "down"):
            dim = 1 if leaf == "down" else 0                # feed-forward width rounded up to eight with zeros
            pad = round_up(w.shape[dim], 8) - w.shape[dim]
            if pad:
                w = torch.nn.functional.pad(w, (0, pad) if dim == 1 else (0, 0, 0, pad))
            return [(f"{base}.{leaf}_proj.weight", w)]
        return [(name, w)]

    def init_random(self, std=0.02, seed=0):
        super().init_random(std, seed)
        for name, t in self.named_params():
            if name.endswith(".a2.b"):
                t.fill_(4.0)                                # decays near one
            elif t.dim() == 1:
                t.fill_(1.0)

    # ------------------------------------------------------------------ forward
    def forward(self, tokens, positions, meta, kv_caches, embeds=None):
        """tokens, positions [T] int64 -> final-norm hidden states [T, width] in the model's dtype."""
        x, y, eps = None, None, self.args.rms_norm_eps
        for layer, kv in zip(self.layers, kv_caches):
            if x is None:
                x, h = residual_update(None, self.embed, rows=tokens, w_out=layer.norm1, eps=eps)
            else:
                _, h = residual_update(x, y, w=side_norm, w_out=layer.norm1, eps=eps)
            y = layer(x, h, tokens, self.side_table, positions, meta, kv, self.state.layers[layer.idx])
            side_norm = layer.side.norm
        return residual_update(x, y, w=side_norm, w_out=self.final_norm, eps=eps)[1]

    def logits(self, hidden_rows):
        return self.lm_head(hidden_rows)

    def logits_local(self, hidden_rows):
        return self.lm_head.forward_local(hidden_rows)

    def gather_logits(self, local):
        return self.lm_head.gather(local)

    def greedy_from_local(self, local):
        return self.lm_head.greedy_from_local(local)

    __call__ = forward


@register_model("femirax", "Femirax", kernel_sources=FemiraxCausalLM.kernel_sources)
def build_femirax(args, dtype, device, ps):
    return FemiraxCausalLM(args, dtype, device, ps)
