"""Sublayers of hybrid decoders over an fp32 residual stream, with their constants as parameters: decayed linear
attention (per-head or per-channel decay), the gated delta rule with channel decays, exponentially gated matrix memory,
attention whose values are its keys, windowed attention with an output gate, a gated per-token side input.

Each mixer names its tensors as a checkpoint does (loader names relative to the mixer) and exposes
  width_parts()   the projections it needs of its input, which the owner fuses into one GEMM,
  forward(rows, meta, ...)  from those projection rows to the mixer's output.
Residual, norms, rotary angles, scores, decays and states are fp32; projections run in the model's dtype.
"""
from __future__ import annotations

from typing import Dict, List, Tuple

import torch

from .. import ops
from ..ops.delta_rule import ChannelDelta
from ..ops.head_norm import head_gate
from ..ops.linear_attn import LinearAttention
from ..ops.mlstm import MatrixMemory
from ..ops.residual import gelu_mul_rows
from .layers import AttentionMetadata, Linear, Module, RotaryEmbedding


def round_up(n, m):
    return (n + m - 1) // m * m


class FusedProjection(Module):
    """Several projections of one input as one GEMM.  `parts`: (loader name, rows); every part starts at a multiple of
    eight columns of the output (16-byte aligned rows for the kernels behind it; the gaps are zero weights).  `biased`:
    the parts with a bias (loader name + ".b").  `f32`: the result stays fp32 (few columns: router logits, gates)."""

    def __init__(self, in_f: int, parts: List[Tuple[str, int]], dtype, device, biased=(), f32=False):
        super().__init__()
        self.f32 = f32
        self.at: Dict[str, Tuple[int, int]] = {}
        off = 0
        for name, n in parts:
            self.at[name] = (off, n)
            off += round_up(n, 8)
        self.weight = torch.zeros(off, in_f, dtype=dtype, device=device)
        self._params["weight"] = self.weight
        for name, (o, n) in self.at.items():
            self._loaders[name] = lambda w, o=o, n=n: self.weight[o:o + n].copy_(w.to(self.weight.dtype))
        self.bias = None
        if biased:
            self.bias = self._params["bias"] = torch.zeros(off, dtype=dtype, device=device)
            for name in biased:
                o, n = self.at[name]
                self._loaders[name + ".b"] = lambda w, o=o, n=n: self.bias[o:o + n].copy_(w.to(self.bias.dtype))

    def named_loaders(self, prefix=""):
        # the parts carry the names of the owner's checkpoint tensors
        owner = prefix[: prefix.rindex(".", 0, -1) + 1] if "." in prefix[:-1] else ""
        for n, f in self._loaders.items():
            yield owner + n, f

    def forward(self, x):
        return ops.linear_f32(x, self.weight, self.bias) if self.f32 else ops.linear(x, self.weight, self.bias)

    def part(self, rows, name, padded=False):
        """Columns of one part; `padded`: with the zero columns behind it."""
        o, n = self.at[name]
        return rows[:, o:o + (round_up(n, 8) if padded else n)]

    __call__ = forward


class OutProjection(Module):
    """y = x W^T where x may be wider than the checkpoint's W: heads stored zero-padded (`head`, `head_pad`)."""

    def __init__(self, heads, head, head_pad, out_f, dtype, device):
        super().__init__()
        self.weight = torch.zeros(out_f, heads * head_pad, dtype=dtype, device=device)

        def load(w):
            self.weight.view(out_f, heads, head_pad)[:, :, :head].copy_(w.view(out_f, heads, head).to(dtype))

        self._params["weight"] = self.weight
        self._loaders["weight"] = load

    def forward(self, x):
        return ops.linear(x, self.weight)

    __call__ = forward


class LinearAttentionMixer(Module):
    """Multi-head linear attention with a decaying state and gated output: retention (`decay`: one constant per head,
    rotated q and k) or per-channel decay (`rank` > 0: low-rank projection a1, a2 and bias a2.b, temperature tau)."""

    def __init__(self, hidden, heads, dk, dv, eps, dtype, device, decay=None, rank=0, tau=1.0, q_scale=1.0, k_scale=1.0,
                 rope: RotaryEmbedding = None, norm_weight=False, prefix=""):
        super().__init__()
        self.prefix, self.state_shape = prefix, (heads, dk, dv)
        self.heads, self.dv = heads, dv
        self.parts = [("q", heads * dk), ("k", heads * dk), ("v", heads * dv), ("g", heads * dv)]
        op = LinearAttention(heads, dk, dv, q_scale=q_scale, k_scale=k_scale, eps=eps)
        if decay is not None:
            d = torch.tensor([float(x) for x in decay], dtype=torch.float64)
            if d.numel() != heads or bool((d < 0).any()) or bool((d > 1).any()):
                raise ValueError(f"retention needs {heads} decays in [0, 1]")
            op.log_decay = torch.log(d.clamp_min(1e-300)).to(torch.float32).to(device)
        else:
            self.parts.append(("a1", rank))
            op.a2 = self.add_param("a2", torch.zeros(heads * dk, rank, dtype=dtype, device=device))
            op.a2_bias = self.add_param("a2.b", torch.zeros(heads * dk, dtype=dtype, device=device))
            op.inv_tau = 1.0 / float(tau)
        if rope is not None:
            op.cos_sin, op.rot, op.interleaved = rope.cos_sin, rope.rot_dim, rope.interleaved
        if norm_weight:
            op.norm_w = self.add_param("norm", torch.ones(dv, dtype=dtype, device=device))
        self.op = op
        self.o = self.add_module("o", Linear(heads * dv, hidden, False, dtype, device))

    def width_parts(self):
        return [(self.prefix + n, w) for n, w in self.parts]

    def forward(self, fused: FusedProjection, rows, positions, meta: AttentionMetadata, state):
        p = {n: fused.part(rows, self.prefix + n) for n, _ in self.parts}
        nd, T = meta.n_decode, rows.shape[0]
        slots, r = meta.state_slots, p.get("a1")
        alloc = torch.zeros if meta.padded or not rows.is_cuda else torch.empty
        out = alloc((T, self.heads * self.dv), dtype=rows.dtype, device=rows.device)
        if nd > 0:
            self.op.decode(state, slots[:nd], meta.kv_lens[:nd], positions[:nd], p["q"][:nd], p["k"][:nd], p["v"][:nd],
                           g=p["g"][:nd], r=r[:nd] if r is not None else None, out=out[:nd])
        if meta.n_prefill > 0:
            self.op.prefill(state, slots[nd:], meta.cu_q[nd:], meta.kv_lens[nd:], positions, p["q"], p["k"], p["v"],
                            g=p["g"], r=r, out=out, row0=nd, padded=meta.padded, max_q_len=meta.max_q_len)
        return self.o(out)

    __call__ = forward


class KeyValueAttention(Module):
    """Causal GQA whose values are the keys as projected (before rotation and norm: no value projection); q and k are
    rotated and then divided by their root mean square per head."""

    def __init__(self, hidden, heads, kv_heads, d, scale, eps, dtype, device, rope: RotaryEmbedding = None, prefix=""):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("the query heads must be a multiple of the key/value heads")
        self.prefix, self.heads, self.kv_heads, self.d = prefix, heads, kv_heads, d
        self.scale, self.eps, self.rope = float(scale), eps, rope
        self.d_pad = ops.attention_head_size(d)
        self.o = self.add_module("o_pad", OutProjection(heads, d, self.d_pad, hidden, dtype, device))

    def named_loaders(self, prefix=""):
        for n, f in super().named_loaders(prefix):
            yield n.replace("o_pad.weight", "o.weight"), f

    def width_parts(self):
        return [(self.prefix + "q", self.heads * self.d), (self.prefix + "k", self.kv_heads * self.d)]

    def kv_geometry(self):
        return (2, self.kv_heads, self.d_pad)

    def forward(self, fused: FusedProjection, rows, positions, meta: AttentionMetadata, k_cache, v_cache):
        q, k = fused.part(rows, self.prefix + "q"), fused.part(rows, self.prefix + "k")
        rope = self.rope
        q = ops.rope_norm_kv_write(q, k, k, self.heads, self.kv_heads, self.d, positions, rope.cos_sin if rope else None,
                                   rope.rot_dim if rope else 0, meta.slots, k_cache, v_cache, eps=self.eps,
                                   interleaved=rope.interleaved if rope else False)
        T, nd = q.shape[0], meta.n_decode
        out = (torch.zeros if meta.padded else torch.empty)(q.shape, dtype=q.dtype, device=q.device)
        if q.is_cuda and (q.dtype != torch.bfloat16 or self.d_pad not in (64, 128, 256)):
            ops.paged_attention_generic(q, k_cache, v_cache, meta.block_table, meta.cu_q, meta.kv_lens, self.scale, out=out)
        else:
            if nd > 0:
                ops.paged_decode_attention(q[:nd], k_cache, v_cache, meta.block_table[:nd], meta.kv_lens[:nd], self.scale,
                                           out=out[:nd])
            if meta.n_prefill > 0:
                ops.paged_prefill_attention(q, k_cache, v_cache, meta.block_table[nd:], meta.cu_q[nd:], meta.kv_lens[nd:],
                                            meta.max_q_len, self.scale, causal=True, out=out)
        return self.o(out.view(T, self.heads * self.d_pad))

    __call__ = forward


class WindowAttention(Module):
    """GQA over a sliding window: biases on q, k and v, rotary positions on the first elements of every q and k head, value
    heads of a size of their own, and (`gate`) outputs multiplied by the sigmoid of a projection of the same input."""

    def __init__(self, hidden, heads, kv_heads, d, dv, scale, window, dtype, device, rope: RotaryEmbedding = None, gate=True):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("the query heads must be a multiple of the key/value heads")
        if int(window) <= 0:
            raise ValueError("a sliding window holds at least the token itself")
        self.heads, self.kv_heads, self.d, self.dv = heads, kv_heads, d, dv
        self.scale, self.window, self.rope, self.gate = float(scale), int(window), rope, gate
        self.d_pad = ops.attention_head_size(max(d, dv))
        self.o = self.add_module("o", Linear(heads * dv, hidden, False, dtype, device))
        self.biased = ("q", "k", "v")

    def width_parts(self):
        return [("q", self.heads * self.d), ("k", self.kv_heads * self.d), ("v", self.kv_heads * self.dv)] + \
            ([("g", self.heads * self.dv)] if self.gate else [])

    def small_parts(self):
        return []

    def kv_geometry(self):
        return (2, self.kv_heads, self.d_pad)

    def state_parts(self):
        return None

    def forward(self, fused: FusedProjection, rows, small, positions, meta: AttentionMetadata, kv, state):
        q, k, v = (fused.part(rows, n) for n in "qkv")
        rope, (k_cache, v_cache) = self.rope, kv
        q = ops.rope_norm_kv_write(q, k, v, self.heads, self.kv_heads, self.d, positions, rope.cos_sin if rope else None,
                                   rope.rot_dim if rope else 0, meta.slots, k_cache, v_cache, unit_norm=False)
        nd = meta.n_decode
        out = (torch.zeros if meta.padded else torch.empty)(q.shape, dtype=q.dtype, device=q.device)
        if q.is_cuda and (q.dtype != torch.bfloat16 or self.d_pad not in (64, 128, 256)):
            ops.paged_attention_generic(q, k_cache, v_cache, meta.block_table, meta.cu_q, meta.kv_lens, self.scale, out=out,
                                        window=self.window)
        else:
            if nd > 0:
                # a window bounds the keys of a row: splitting them further than a few hundred apiece costs more than it gives
                splits = min(ops.decode_splits(nd, self.kv_heads, self.heads // self.kv_heads), max(1, self.window // 256))
                ops.paged_decode_attention(q[:nd], k_cache, v_cache, meta.block_table[:nd], meta.kv_lens[:nd], self.scale,
                                           out=out[:nd], window=self.window, splits=splits)
            if meta.n_prefill > 0:
                ops.paged_prefill_attention(q, k_cache, v_cache, meta.block_table[nd:], meta.cu_q[nd:], meta.kv_lens[nd:],
                                            meta.max_q_len, self.scale, causal=True, window=self.window, out=out)
        if self.gate:
            return self.o(head_gate(out, fused.part(rows, "g"), self.dv))
        return self.o(out[..., : self.dv].reshape(out.shape[0], self.heads * self.dv))

    __call__ = forward


class DeltaRuleMixer(Module):
    """Gated delta rule with a decay per key channel (ops/delta_rule.py): short convolutions on q, k and v, unit q and k,
    low-rank decay (a1, a2, dt_bias, A_log) and output gate (g1, g2), a norm weight shared by the heads."""

    def __init__(self, hidden, heads, kv_heads, dk, dv, taps, decay_rank, gate_rank, eps, dtype, device):
        super().__init__()
        if heads % kv_heads:
            raise ValueError("the value heads must be a multiple of the query/key heads")
        op = self.op = ChannelDelta(heads, kv_heads, dk, dv, taps, q_scale=dk ** -0.5, eps=eps)
        self.parts = [("q", kv_heads * dk), ("k", kv_heads * dk), ("v", heads * dv), ("a1", decay_rank), ("g1", gate_rank)]
        op.conv_w = self._params["conv"] = torch.zeros(taps, op.channels, dtype=dtype, device=device)
        at = 0
        for n, c in self.parts[:3]:
            self._loaders[n + ".conv"] = lambda w, o=at, c=c: op.conv_w[:, o:o + c].copy_(w.reshape(c, taps).T.to(dtype))
            at += c
        op.a2 = self.add_param("a2", torch.zeros(heads * dk, decay_rank, dtype=dtype, device=device))
        op.dt_bias = self.add_param("dt_bias", torch.zeros(heads * dk, dtype=dtype, device=device))
        op.a_log = self.add_param("A_log", torch.zeros(heads, dtype=dtype, device=device))
        op.norm_w = self.add_param("norm", torch.ones(dv, dtype=dtype, device=device))
        self.g2 = self._params["g2"] = torch.zeros(heads * dv, round_up(gate_rank, 8), dtype=dtype, device=device)
        self._loaders["g2"] = lambda w: self.g2[:, :gate_rank].copy_(w.to(dtype))
        self.o = self.add_module("o", Linear(heads * dv, hidden, False, dtype, device))
        self.biased = ()

    def width_parts(self):
        return self.parts

    def small_parts(self):
        return [("b", self.op.heads, False)]

    def kv_geometry(self):
        return None

    def state_parts(self):
        op = self.op
        return {"S": ((op.heads, op.dk, op.dv), None), "conv": ((op.taps, op.channels), op.conv_w.dtype)}

    def forward(self, fused: FusedProjection, rows, small, positions, meta: AttentionMetadata, kv, state):
        q, k, v, r = (fused.part(rows, n) for n in ("q", "k", "v", "a1"))
        gate = ops.linear(fused.part(rows, "g1", padded=True), self.g2)
        nd, T, slots, zb = meta.n_decode, rows.shape[0], meta.state_slots, small["b"]
        alloc = torch.zeros if meta.padded or not rows.is_cuda else torch.empty
        out = alloc((T, self.op.heads * self.op.dv), dtype=rows.dtype, device=rows.device)
        if nd > 0:
            self.op.decode(state["S"], state["conv"], slots[:nd], meta.cu_q[:nd + 1], meta.kv_lens[:nd], q[:nd], k[:nd], v[:nd],
                           r[:nd], zb[:nd], gate[:nd], out[:nd])
        if meta.n_prefill > 0:
            self.op.prefill(state["S"], state["conv"], slots[nd:], meta.cu_q[nd:], meta.kv_lens[nd:], q, k, v, r, zb, gate, out,
                            row0=nd, padded=meta.padded, max_q_len=meta.max_q_len)
        return self.o(out)

    __call__ = forward


class MatrixMemoryMixer(Module):
    """Matrix memory with exponential gates (ops/mlstm.py): one input and one forget gate per head from fp32 projections
    with biases, outputs normed per head, weighted, gated."""

    def __init__(self, hidden, heads, dk, dv, cap, eps, dtype, device):
        super().__init__()
        op = self.op = MatrixMemory(heads, dk, dv, float(cap), q_scale=dk ** -0.5, eps=eps)
        op.norm_w = self.add_param("norm", torch.ones(heads * dv, dtype=dtype, device=device))
        self.o = self.add_module("o", Linear(heads * dv, hidden, False, dtype, device))
        self.biased = ()

    def width_parts(self):
        op = self.op
        return [("q", op.heads * op.dk), ("k", op.heads * op.dk), ("v", op.heads * op.dv), ("g", op.heads * op.dv)]

    def small_parts(self):
        return [("i", self.op.heads, True), ("f", self.op.heads, True)]

    def kv_geometry(self):
        return None

    def state_parts(self):
        op, f32 = self.op, torch.float32
        return {"S": ((op.heads, op.dk, op.dv), None), "n": ((op.heads, op.dk), f32), "m": ((op.heads,), f32)}

    def forward(self, fused: FusedProjection, rows, small, positions, meta: AttentionMetadata, kv, state):
        q, k, v, gate = (fused.part(rows, n) for n in "qkvg")
        nd, T, slots, zi, zf = meta.n_decode, rows.shape[0], meta.state_slots, small["i"], small["f"]
        alloc = torch.zeros if meta.padded or not rows.is_cuda else torch.empty
        out = alloc((T, self.op.heads * self.op.dv), dtype=rows.dtype, device=rows.device)
        if nd > 0:
            self.op.decode(state, slots[:nd], meta.cu_q[:nd + 1], meta.kv_lens[:nd], q[:nd], k[:nd], v[:nd], zi[:nd], zf[:nd],
                           gate[:nd], out[:nd])
        if meta.n_prefill > 0:
            self.op.prefill(state, slots[nd:], meta.cu_q[nd:], meta.kv_lens[nd:], q, k, v, zi, zf, gate, out, row0=nd,
                            padded=meta.padded)
        return self.o(out)

    __call__ = forward


class TokenSideInput(Module):
    """A per-token input beside the sublayers: y = proj(gelu_tanh(gate x) * e) with e the layer's columns of a table row
    picked by the token; the caller adds y / rms(y) * norm to the residual."""

    def __init__(self, hidden, dim, col0, dtype, device):
        super().__init__()
        self.dim, self.col0 = dim, col0
        pad = round_up(dim, 8)
        self.gate = torch.zeros(pad, hidden, dtype=dtype, device=device)
        self.proj = torch.zeros(hidden, pad, dtype=dtype, device=device)
        self._params.update(gate=self.gate, proj=self.proj)
        self._loaders["gate"] = lambda w: self.gate[:dim].copy_(w.to(dtype))
        self._loaders["proj"] = lambda w: self.proj[:, :dim].copy_(w.to(dtype))
        self.norm = self.add_param("norm", torch.ones(hidden, dtype=dtype, device=device))

    def forward(self, xb, table, tokens):
        g = gelu_mul_rows(ops.linear(xb, self.gate), table, tokens, self.col0, self.dim)
        return ops.linear(g, self.proj)

    __call__ = forward
