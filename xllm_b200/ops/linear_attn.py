"""Linear attention with a decaying matrix state: S_t = diag(a_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.

`LinearAttention` carries the constants of one layer (head sizes, decay, rotary table, scales, output norm); its
methods take column blocks of the layer's projection rows as they are.  On CUDA everything runs in
csrc/kernels/linear_attn.cu; CPU tensors take the same arithmetic in tensor ops."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from ._lib import F, I, L, P, check, ptr, stream
from .head_norm import head_norm_gate

_lib.register_signature("xllm_linattn", [P] * 9 + [L, P, L, P, P, P, P, P, P, L] + [I] * 8 + [F] * 4 + [I, I, P, P, I, I, I, I, P])

_DT = {torch.bfloat16: 0, torch.float32: 1}


@dataclass
class LinearAttention:
    heads: int
    dk: int
    dv: int
    q_scale: float = 1.0
    k_scale: float = 1.0
    # decay: one constant per head (fp32 [heads], its logarithm) or, per token and key channel,
    # sigmoid(a2 r + a2_bias) ** inv_tau with r the low-rank column block of the projection row
    log_decay: Optional[torch.Tensor] = None
    a2: Optional[torch.Tensor] = None
    a2_bias: Optional[torch.Tensor] = None
    inv_tau: float = 1.0
    # rotary positions on the first `rot` elements of every q and k head
    cos_sin: Optional[torch.Tensor] = None
    rot: int = 0
    interleaved: bool = False
    in_silu: bool = False            # q, k and v pass through silu first
    # `rows`: the heads of a token are normed together over all their elements and gated with the sigmoid of g; otherwise
    # every head is finished alone and gated with silu(g)
    rows: bool = False
    # output of a head: divided by its root mean square, times the weight [dv] when there is one (`rows`: [heads dv])
    unit_norm: bool = True
    norm_w: Optional[torch.Tensor] = None
    eps: float = 1e-6

    def _launch(self, mode, state, slots, cu_q, kv_lens, positions, q, k, v, g, r, out, out_ld, n_seqs, seg=(None, None, 16, 1), finish=False):
        ld = q.stride(0)
        for t in (k, v, g, r):
            assert t is None or (t.stride(0) == ld and t.stride(1) == 1 and t.dtype == q.dtype)
        assert q.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
        assert state.shape[1:] == (self.heads, self.dk, (self.dv + 3) // 4 * 4)
        assert slots.dtype == torch.int32 and kv_lens.dtype == torch.int32 and slots.shape[0] >= n_seqs
        channel = self.log_decay is None
        use_rope = self.rot > 0
        assert not use_rope or (positions.dtype == torch.int64 and self.cos_sin.shape[1] == self.rot)
        check(_lib.load().xllm_linattn(
            ptr(state), ptr(slots), ptr(cu_q), ptr(kv_lens), ptr(q), ptr(k), ptr(v), ptr(g), ptr(r if channel else None), ld,
            ptr(self.cos_sin if use_rope else None), self.cos_sin.shape[0] if use_rope else 0, ptr(positions),
            ptr(self.log_decay), ptr(self.a2), ptr(self.a2_bias), ptr(self.norm_w), ptr(out), out_ld, n_seqs, self.heads,
            self.dk, self.dv, self.rot, int(self.interleaved), self.a2.shape[1] if channel else 0, int(self.unit_norm),
            self.q_scale, self.k_scale, self.inv_tau, self.eps, _DT[q.dtype], mode, ptr(seg[0]), ptr(seg[1]),
            seg[2], seg[3], int(finish), int(self.in_silu), stream()), "linattn")
        from . import _count
        _count()

    def decode(self, state, slots, kv_lens, positions, q, k, v, g=None, r=None, out=None):
        """One token per sequence (sequence s is row s); returns the finished rows [B, heads * dv].  Rows with a
        negative slot are padding and come out zero."""
        B = slots.shape[0]
        if not q.is_cuda:
            return self._cpu(state, slots, torch.arange(B + 1), kv_lens, positions, q, k, v, r, g, out)
        if out is None:
            out = torch.empty((B, self.heads * self.dv), dtype=q.dtype, device=q.device)
        if self.rows:
            o = torch.empty((B, self.heads, self.dv), dtype=torch.float32, device=q.device)
            self._launch(0, state, slots, None, kv_lens, positions, q, k, v, None, r, o, 0, B)
            return self.finish(o, g, out)
        self._launch(0, state, slots, None, kv_lens, positions, q, k, v, g, r, out, out.stride(0), B, finish=True)
        return out

    def prefill(self, state, slots, cu_q, kv_lens, positions, q, k, v, g=None, r=None, out=None, row0=0, padded=False,
                token_by_token=False, max_q_len=None):
        """Prompt rows of several sequences (absolute token rows cu_q, all at or behind row0); fills rows [row0, T) of
        `out` [T, heads * dv].  `padded`: rows outside every sequence exist and must come out finite.
        `max_q_len`: the most rows any sequence has (default: all rows).  `token_by_token`: the fp32 recurrence instead of the chunked form."""
        n = slots.shape[0]
        if not q.is_cuda:
            return self._cpu(state, slots, cu_q, kv_lens, positions, q, k, v, r, g, out)
        T = q.shape[0]
        if out is None:
            out = torch.empty((T, self.heads * self.dv), dtype=q.dtype, device=q.device)
        chunked = q.dtype == torch.bfloat16 and self.dk <= 256 and not token_by_token and \
            (self.a2 is None or self.a2.shape[1] <= 64)
        fused = chunked and self.dv <= 128 and not self.rows
        seg = self._segments(T, n, max_q_len or T, q.device) if chunked else (None, None, 16, 1)
        if fused:
            self._launch(1, state, slots, cu_q, kv_lens, positions, q, k, v, g, r, out, out.stride(0), n, seg=seg, finish=True)
            return out
        o = (torch.zeros if padded else torch.empty)((T, self.heads, self.dv), dtype=torch.float32, device=q.device)
        self._launch(1 if chunked else 2, state, slots, cu_q, kv_lens, positions, q, k, v, None, r, o, 0, n, seg=seg)
        self.finish(o[row0:], g[row0:] if g is not None else None, out[row0:])
        return out

    def _segments(self, T, n_seqs, max_q_len, device):
        """(states, decays, segment length, segments per sequence): long prompts are cut so that the CTAs of one launch
        (heads x value slices x segments) fill the GPU about twice; short ones stay whole."""
        ctas = self.heads * -(-self.dv // 128)
        length = min(1024, max(128, -(-T * ctas // 592)))
        length = -(-length // 64) * 64
        segs = -(-max_q_len // length)
        if segs == 1:
            return None, None, length, 1
        m = T // length + n_seqs + 1
        st = torch.empty((m, self.heads, self.dk, (self.dv + 3) // 4 * 4), dtype=torch.float32, device=device)
        return st, torch.empty((m, self.heads, self.dk), dtype=torch.float32, device=device), length, segs

    def finish(self, o, g, out):
        """Norm, weight and gate of raw fp32 outputs o [T, heads, dv]."""
        if self.rows:
            return head_norm_gate(o.view(o.shape[0], 1, -1), out, g=g, w=self.norm_w, unit_norm=self.unit_norm, act="sigmoid",
                                  eps=self.eps)
        return head_norm_gate(o, out, g=g, w=self.norm_w, unit_norm=self.unit_norm, eps=self.eps)

    # ------------------------------------------------------------------ tensor-op form
    def _rope(self, x, positions):
        if self.rot == 0:
            return x
        cs = self.cos_sin[positions]
        c, s = cs[:, None, : self.rot // 2], cs[:, None, self.rot // 2:]
        xr = x[..., : self.rot]
        if self.interleaved:
            a, b = xr[..., 0::2], xr[..., 1::2]
            y = torch.stack([a * c - b * s, b * c + a * s], dim=-1).flatten(-2)
        else:
            a, b = xr.chunk(2, dim=-1)
            y = torch.cat([a * c - b * s, b * c + a * s], dim=-1)
        return torch.cat([y, x[..., self.rot:]], dim=-1)

    def _cpu(self, state, slots, cu_q, kv_lens, positions, q, k, v, r, g, out):
        H, dk, dv = self.heads, self.dk, self.dv
        T = q.shape[0]
        res = out if out is not None else torch.zeros(T, H * dv, dtype=q.dtype)
        enter = (lambda t: torch.nn.functional.silu(t.float())) if self.in_silu else (lambda t: t.float())
        qf = self._rope(enter(q).reshape(T, H, dk), positions) * self.q_scale
        kf = self._rope(enter(k).reshape(T, H, dk), positions) * self.k_scale
        vf = enter(v).reshape(T, H, dv)
        if self.log_decay is None:
            z = r.float() @ self.a2.float().T + self.a2_bias.float()
            less = torch.expm1(torch.nn.functional.logsigmoid(z) * self.inv_tau).view(T, H, dk)     # a - 1
        else:
            less = torch.expm1(self.log_decay).view(1, H, 1).expand(T, H, dk)
        for i in range(slots.shape[0]):
            b, e, slot = int(cu_q[i]), int(cu_q[i + 1]), int(slots[i])
            if slot < 0 or e <= b:
                continue
            S = state[slot, :, :, :dv].clone() if int(kv_lens[i]) != e - b else torch.zeros(H, dk, dv)
            o = torch.empty(e - b, H, dv)
            for t in range(b, e):
                S = S + less[t][:, :, None] * S + kf[t][:, :, None] * vf[t][:, None, :]
                o[t - b] = torch.einsum("hkv,hk->hv", S, qf[t])
            state[slot, :, :, :dv] = S
            if self.rows:
                self.finish(o, g[b:e] if g is not None else None, res[b:e])
                continue
            if self.unit_norm:
                o = o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + self.eps)
            if self.norm_w is not None:
                o = o * self.norm_w.float()
            o = o.reshape(e - b, H * dv)
            if g is not None:
                o = o * torch.nn.functional.silu(g[b:e].float())
            res[b:e] = o.to(res.dtype)
        return res
