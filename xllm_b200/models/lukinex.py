"""Lukinex: a small hybrid decoder with a norm before and behind every sublayer.

Layers come in any order from the configuration: `parallel` (windowed attention behind short convolutions, its scores softly
capped, beside lightning attention; the two outputs are normalised over the width and averaged), `attention` (windowed, q and k
heads normed) or `latent_attention` (no positions, one cached latent per token; a layer may read the latents of an earlier
one).  Windows keep the first tokens visible.  Feed-forwards are mixtures of clamped experts with a shared one, or none.  The
residual is fp32 throughout.

    x <- x + norm1b(mixer(norm1 x));   x <- x + norm2b(ff(norm2 x))

The mechanisms live in models/mixers.py and models/qwen_moe.py; this file reads the configuration and strings them together so
that every residual update is one launch with the norms on both of its sides (ops/residual.py).  There is no counterpart in
the reference's zoo (xllm/models/llm/).
"""
from __future__ import annotations

import dataclasses

import torch

from ..ops.glu import ClampedGLU
from ..ops.residual import residual_update
from ..parallel.state import single
from .layers import LMHead, Module, RotaryEmbedding
from .mixers import FusedProjection, KeptWindowAttention, LatentAttention, LinearAttentionMixer, round_up
from .qwen_moe import SparseMoeBlock
from .registry import register_model
from .state import RecurrentStatePool


def _rope(rot, args, device):
    if int(rot["dims"]) == 0:
        return None
    s = rot.get("scaling")
    return RotaryEmbedding(int(rot["dims"]), args.max_position_embeddings, float(rot["base"]),
                           {"rope_type": "linear", "factor": s["factor"]} if s else None, device)


def _window_attention(m, args, dtype, device, **kw):
    size, keep = int(m["mask"]["size"]), int(m["mask"].get("keep_first", 0))
    if size <= 0:
        raise ValueError("a sliding window holds at least the token itself")
    return KeptWindowAttention(args.hidden_size, int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), m["scale"],
                               size, keep, args.rms_norm_eps, dtype, device, rope=_rope(m["rot"], args, device), **kw)


class LukinexLayer(Module):
    def __init__(self, args, idx, dtype, device):
        super().__init__()
        spec, eps, W = args.extra["layers"][idx], args.rms_norm_eps, args.hidden_size
        m, self.idx, self.eps = spec["mixer"], idx, eps
        norm = lambda name: self.add_param(name, torch.ones(W, dtype=dtype, device=device))
        self.norm1, self.norm1b = norm("norm1"), norm("norm1b")
        self.cache_of, self.linear = idx, None       # the layer whose paged cache this one reads
        if spec["type"] == "parallel":
            mix, l, r = self.add_module("mix", Module()), m["left"], m["right"]
            self.mixer = mix.add_module("left", _window_attention(l, args, dtype, device, softcap=float(l["softcap"]),
                                                                  taps=int(l["conv"]), bias=True, prefix="left."))
            self.linear = mix.add_module("right", LinearAttentionMixer(
                W, int(r["heads"]), int(r["dim"]), int(r["vdim"]), eps, dtype, device, decay=r["decay"], norm_weight=True,
                prefix="right.", in_silu=True, row_norm=True))
            self.left_out = mix.add_param("left.out", torch.ones(W, dtype=dtype, device=device))
            self.right_out = mix.add_param("right.out", torch.ones(W, dtype=dtype, device=device))
            parts = self.mixer.width_parts() + self.linear.width_parts()
        elif spec["type"] == "attention":
            mix = self.mixer = self.add_module("mix", _window_attention(m, args, dtype, device, qk_norm=True))
            parts = mix.width_parts()
        elif spec["type"] == "latent_attention":
            source = m.get("kv_from")
            if source is not None:
                self.cache_of = int(source)
                other = args.extra["layers"][self.cache_of] if 0 <= self.cache_of < idx else {}
                if other.get("type") != "latent_attention" or other["mixer"].get("kv_from") is not None or \
                        other["mixer"]["kv_rank"] != m["kv_rank"]:
                    raise ValueError(f"layer {idx}: layer {source} has no latents of {m['kv_rank']} values for it")
            mix = self.mixer = self.add_module("mix", LatentAttention(
                W, int(m["heads"]), int(m["dim"]), int(m["vdim"]), int(m["q_rank"]), int(m["kv_rank"]), m["scale"], eps, dtype,
                device, own_latents=source is None))
            parts = mix.width_parts()
        else:
            raise ValueError(f"unknown mixer type {spec['type']!r} of layer {idx}")
        self.proj = mix.add_module("in", FusedProjection(W, parts, dtype, device, biased=self.mixer.biased))
        self.mlp, f = None, spec.get("mlp")
        if f is not None:
            if f["kind"] != "moe":
                raise ValueError(f"unknown feed-forward kind {f['kind']!r} of layer {idx}")
            E, K, s = int(f["router"]["experts"]), int(f["router"]["top"]), f["shared"]
            if not 0 < K <= E:
                raise ValueError(f"layer {idx}: {E} experts do not hold {K}")
            self.norm2, self.norm2b = norm("norm2"), norm("norm2b")
            self.router = self.add_module("small", FusedProjection(W, [("mlp.router", E)], dtype, device, f32=True))
            # the tensor-core products with the activation in their epilogues take widths in steps of 64
            self.ff_to = 64 if torch.device(device).type == "cuda" and dtype == torch.bfloat16 else 1
            a = dataclasses.replace(
                args, num_experts=E, num_experts_per_tok=K, moe_intermediate_size=round_up(int(f["expert"]["ff"]), self.ff_to),
                scoring_func="softmax", n_group=1, topk_group=1, norm_topk_prob=True, routed_scaling_factor=1.0,
                router_bias=False, n_shared_experts=1, shared_expert_intermediate_size=round_up(int(s["ff"]), self.ff_to),
                fp8_execution=False)
            self.mlp = self.add_module("mlp", SparseMoeBlock(a, dtype, device, own_router=False,
                                                             act=ClampedGLU(float(f["expert"]["limit"])),
                                                             shared_act=ClampedGLU(float(s["limit"]))))

    def state_parts(self):
        parts = dict(self.mixer.state_parts())
        if self.linear is not None:
            parts["S"] = (self.linear.state_shape, None)
        return parts

    def forward(self, x, h, positions, meta, kv, state, w_out):
        """x: fp32 residual (updated in place); h: norm1(x).  Returns the residual through the norm w_out of what follows."""
        rows, eps = self.proj(h), self.eps
        a = self.mixer(self.proj, rows, positions, meta, kv, state)
        after = w_out if self.mlp is None else self.norm2
        if self.linear is not None:
            b = self.linear(self.proj, rows, positions, meta, state["S"])
            _, h = residual_update(x, a, w=self.left_out, y2=b, w2=self.right_out, coef=0.5, w_sum=self.norm1b, w_out=after, eps=eps)
        else:
            _, h = residual_update(x, a, w=self.norm1b, w_out=after, eps=eps)
        if self.mlp is None:
            return h
        y = self.mlp(h, logits=self.router.part(self.router(h), "mlp.router"))
        return residual_update(x, y, w=self.norm2b, w_out=w_out, eps=eps)[1]

    __call__ = forward


class LukinexCausalLM(Module):
    state_on_device = True          # state slots are a device input of the step: graphs capture it
    supports_graph = True
    supports_prefill_graph = True
    # the kernel sources a process that runs nothing but this model needs
    kernel_sources = ("gemm_tcgen05", "activation", "attn_decode", "attn_prefill", "attn_prefill_tc", "attn_generic",
                      "linear_attn", "head_norm", "mla", "proj_f32", "moe", "residual", "rope_norm_kv", "misc", "sampling")
    fused_tp = False

    def __init__(self, args, dtype=torch.bfloat16, device="cpu", ps=None):
        super().__init__()
        self.args, self.ps, self.dtype, self.device = args, ps or single(), dtype, torch.device(device)
        if self.ps.tp_size != 1:
            raise ValueError("Lukinex runs unsharded (one GPU per replica)")
        W = args.hidden_size
        self.embed = self.add_param("embed", torch.zeros(args.vocab_size, W, dtype=dtype, device=device))
        self.layers = [self.add_module(f"l{i}", LukinexLayer(args, i, dtype, device)) for i in range(args.num_hidden_layers)]
        self.final_norm = self.add_param("final.norm", torch.ones(W, dtype=dtype, device=device))
        self.lm_head = self.add_module("head", LMHead(args.vocab_size, W, dtype, device, self.ps))
        self.needs_state = bool(self._state_shapes())
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

    @property
    def max_prefill_graph_tokens(self):
        """Latent layers with many heads expand the context of longer prompt portions, whose lengths a captured step hides."""
        wide = [l.mixer for l in self.layers if isinstance(l.mixer, LatentAttention) and l.mixer.expand_from is not None and
                l.mixer.heads * l.mixer.width >= 8192]
        return min([m.expand_from for m in wide]) if wide else None

    def _state_shapes(self):
        return {l.idx: l.state_parts() for l in self.layers if l.state_parts()}

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
        if ".mlp." not in base:
            return [(name, w)]
        # gate, up, down of the shared expert or of expert e: its width rounded up with zeros
        owner, _, expert = base.rpartition(".")
        dim, to = 1 if leaf == "down" else 0, self.layers[int(name[1:name.index(".")])].ff_to
        pad = round_up(w.shape[dim], to) - w.shape[dim]
        if pad:
            w = torch.nn.functional.pad(w, (0, pad) if dim == 1 else (0, 0, 0, pad))
        part = "shared_experts" if expert == "shared" else f"experts.{expert[1:]}"
        return [(f"{owner}.{part}.{leaf}_proj.weight", w)]

    def init_random(self, std=0.02, seed=0):
        super().init_random(std, seed)
        for name, t in self.named_params():
            if name.endswith("conv"):
                t[-1] += 1.0
            elif name.endswith((".b", "bias")):
                t.zero_()
            elif t.dim() == 1:
                t.fill_(1.0)

    # ------------------------------------------------------------------ forward
    def forward(self, tokens, positions, meta, kv_caches, embeds=None):
        """tokens, positions [T] int64 -> final-norm hidden states [T, width] in the model's dtype."""
        x, h = residual_update(None, self.embed, rows=tokens, w_out=self.layers[0].norm1, eps=self.args.rms_norm_eps)
        states = self.state.layers if self.state is not None else {}
        for layer, w_out in zip(self.layers, [l.norm1 for l in self.layers[1:]] + [self.final_norm]):
            h = layer(x, h, positions, meta, kv_caches[layer.cache_of], states.get(layer.idx), w_out)
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


@register_model("lukinex", "Lukinex", kernel_sources=LukinexCausalLM.kernel_sources)
def build_lukinex(args, dtype, device, ps):
    return LukinexCausalLM(args, dtype, device, ps)
