"""Vivazen: a small decoder whose residual stream is normed behind every sum.

Layers come in any order from the configuration: `attention` (GQA behind short convolutions, whole rows of q and k normed, unit-norm
values, no positions, softly capped scores, softmax weights mixed across heads) or `latent_attention` (one cached latent and one
rotated key part per token, a sliding window, a sink and an output gate per head).  A layer may use an earlier layer's tensors with a
cache and state of its own (`weights_of`).  Feed-forwards are dense or none.  The residual is fp32 throughout.

    x <- norm1(alpha x + mixer(x));   x <- norm2(alpha x + ff(x))

The norm works on equal parts of the width, each over its own root mean square.  The mechanisms live in models/mixers.py; this file
reads the configuration and strings them together so that every residual update is one launch with its norm and the cast that the
next sublayer reads (ops/residual.py).  There is no counterpart in the reference's zoo (xllm/models/llm/).
"""
from __future__ import annotations

import math

import torch

from ..ops.residual import postnorm_update, residual_update
from ..parallel.state import single
from .layers import DenseMLP, LMHead, Module, RotaryEmbedding
from .mixers import FusedProjection, LatentAttention, TalkingAttention, round_up
from .registry import register_model
from .state import RecurrentStatePool


def _yarn(rot, args, device):
    """Neighbouring elements turn together; low frequencies are divided by the factor, and cos and sin grow with its logarithm."""
    s = rot.get("scaling")
    if s is None:
        return RotaryEmbedding(int(rot["dims"]), args.max_position_embeddings, float(rot["base"]), None, device, interleaved=True)
    return RotaryEmbedding(int(rot["dims"]), args.max_position_embeddings, float(rot["base"]),
                           {"rope_type": "yarn", "factor": float(s["factor"]), "original_max_position_embeddings": s["original"],
                            "beta_fast": s["fast"], "beta_slow": s["slow"],
                            "attention_factor": 0.1 * math.log(float(s["factor"])) + 1.0}, device, interleaved=True)


class VivazenLayer(Module):
    """The tensors of one layer; `forward` runs it on the cache and state of any of the layers that use them."""

    def __init__(self, args, idx, dtype, device):
        super().__init__()
        spec, W = args.extra["layers"][idx], args.hidden_size
        m, self.eps, self.groups, self.alpha = spec["mixer"], args.rms_norm_eps, args.extra["norm_groups"], args.extra["postln_alpha"]
        norm = lambda name: self.add_param(name, torch.ones(W, dtype=dtype, device=device))
        self.norm1 = norm("norm1")
        if spec["type"] == "attention":
            mix = TalkingAttention(W, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), m["scale"], m["softcap"],
                                   m["conv"], self.eps, dtype, device)
        elif spec["type"] == "latent_attention":
            if int(m["mask"]["size"]) <= 0:
                raise ValueError("a sliding window holds at least the token itself")
            if int(m["rot"]["dims"]) != int(m["rot_dim"]) or int(m["rot_dim"]) % 2 or int(m["rot_dim"]) <= 0:
                raise ValueError(f"layer {idx}: the rotated part is rotated whole, in pairs")
            mix = LatentAttention(W, int(m["heads"]), int(m["dim"]), int(m["vdim"]), 0, int(m["kv_rank"]), m["scale"], self.eps, dtype,
                                  device, rope=_yarn(m["rot"], args, device), window=m["mask"]["size"], sink=True, gate=True)
        else:
            raise ValueError(f"unknown mixer type {spec['type']!r} of layer {idx}")
        self.mixer = self.add_module("mix", mix)
        self.proj = mix.add_module("in", FusedProjection(W, mix.width_parts(), dtype, device))
        self.mlp, f = None, spec.get("mlp")
        if f is not None:
            if f["kind"] != "dense":
                raise ValueError(f"unknown feed-forward kind {f['kind']!r} of layer {idx}")
            self.norm2 = norm("norm2")
            # the tensor-core product with the activation in its epilogue takes widths in steps of 64
            self.ff_to = 64 if torch.device(device).type == "cuda" and dtype == torch.bfloat16 else 1
            self.mlp = self.add_module("mlp", DenseMLP(W, round_up(int(f["ff"]), self.ff_to), "gelu_tanh", dtype, device))

    def forward(self, x, h, positions, meta, kv, state, w_out=None):
        """x: fp32 residual (updated in place); h: x in the model's dtype.  Returns the new h, through the norm w_out if given."""
        after = dict(alpha=self.alpha, groups=self.groups, eps=self.eps)
        y = self.mixer(self.proj, self.proj(h), positions, meta, kv, state)
        _, h = postnorm_update(x, y, self.norm1, w_out=w_out if self.mlp is None else None, **after)
        if self.mlp is None:
            return h
        return postnorm_update(x, self.mlp(h), self.norm2, w_out=w_out, **after)[1]

    __call__ = forward


class VivazenCausalLM(Module):
    state_on_device = True          # state slots are a device input of the step: graphs capture it
    supports_graph = True
    supports_prefill_graph = True
    # the kernel sources a process that runs nothing but this model needs
    kernel_sources = ("gemm_tcgen05", "activation", "attn_decode", "attn_prefill", "attn_prefill_tc", "attn_generic", "attn_talk", "head_norm",
                      "mla", "residual", "rope_norm_kv", "misc", "sampling")
    fused_tp = False

    def __init__(self, args, dtype=torch.bfloat16, device="cpu", ps=None):
        super().__init__()
        self.args, self.ps, self.dtype, self.device = args, ps or single(), dtype, torch.device(device)
        if self.ps.tp_size != 1:
            raise ValueError("Vivazen runs unsharded (one GPU per replica)")
        W = args.hidden_size
        if args.extra["norm_groups"] <= 0 or W % args.extra["norm_groups"]:
            raise ValueError(f"a width of {W} has no {args.extra['norm_groups']} equal parts")
        self.embed = self.add_param("embed", torch.zeros(args.vocab_size, W, dtype=dtype, device=device))
        owners = [self._owner(args.extra["layers"], i) for i in range(args.num_hidden_layers)]
        made = {i: self.add_module(f"l{i}", VivazenLayer(args, i, dtype, device)) for i in sorted(set(owners))}
        self.layers = [made[i] for i in owners]
        self.final_norm = self.add_param("final.norm", torch.ones(W, dtype=dtype, device=device))
        self.lm_head = self.add_module("head", LMHead(args.vocab_size, W, dtype, device, self.ps))
        self.needs_state = bool(self._state_shapes())
        self.state = None

    @staticmethod
    def _owner(specs, i):
        """The layer whose tensors layer i uses."""
        seen, spec = set(), specs[i]
        while specs[i].get("weights_of") is not None:
            seen.add(i)
            i = int(specs[i]["weights_of"])
            if not 0 <= i < len(specs) or i in seen:
                raise ValueError(f"layer {i} has no tensors to lend")
        same = lambda s: {k: v for k, v in s.items() if k != "weights_of"}
        if same(specs[i]) != same(spec):
            raise ValueError(f"layer {i} lends its tensors to a layer of other sizes")
        return i

    # ------------------------------------------------------------------ cache and state geometry
    def kv_layout(self):
        """Per layer: (planes, kv heads, head size) of its paged cache."""
        return [l.mixer.kv_geometry() for l in self.layers]

    @property
    def num_kv_heads_local(self):
        return max([g[1] for g in self.kv_layout()] + [1])

    @property
    def head_dim(self):
        return max([g[2] for g in self.kv_layout()] + [64])

    def _state_shapes(self):
        return {i: l.mixer.state_parts() for i, l in enumerate(self.layers) if l.mixer.state_parts()}

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
        if leaf == "o" and base.endswith(".mix"):
            return [(name + ".weight", w)]
        if base.endswith(".mlp") and leaf in ("gate", "up", "down"):
            layer = self.layers[int(name[1:name.index(".")])]
            dim = 1 if leaf == "down" else 0                # feed-forward width rounded up with zeros
            pad = round_up(w.shape[dim], layer.ff_to) - w.shape[dim]
            if pad:
                w = torch.nn.functional.pad(w, (0, pad) if dim == 1 else (0, 0, 0, pad))
            return [(f"{base}.{leaf}_proj.weight", w)]
        return [(name, w)]

    def init_random(self, std=0.02, seed=0):
        super().init_random(std, seed)
        for name, t in self.named_params():
            if name.endswith("conv"):
                t[-1] += 1.0
            elif name.endswith("talk"):
                t += torch.eye(t.shape[0], dtype=t.dtype, device=t.device)
            elif name.endswith("sink"):
                t.zero_()
            elif t.dim() == 1:
                t.fill_(1.0)
        for l in self.layers:
            if isinstance(l.mixer, LatentAttention):
                l.mixer.fill_padding()

    # ------------------------------------------------------------------ forward
    def forward(self, tokens, positions, meta, kv_caches, embeds=None):
        """tokens, positions [T] int64 -> final-norm hidden states [T, width] in the model's dtype."""
        x, h = residual_update(None, self.embed, rows=tokens)
        states = self.state.layers if self.state is not None else {}
        for i, layer in enumerate(self.layers):
            w_out = self.final_norm if i + 1 == len(self.layers) else None
            h = layer(x, h, positions, meta, kv_caches[i], states.get(i), w_out)
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


@register_model("vivazen", "Vivazen", kernel_sources=VivazenCausalLM.kernel_sources)
def build_vivazen(args, dtype, device, ps):
    return VivazenCausalLM(args, dtype, device, ps)
