"""Gated delta rule with a decay per key channel: S <- diag(g) S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.

`ChannelDelta` carries the constants and small weights of one layer; its methods take column blocks of the layer's
projection rows as they are (before the short convolutions).  On CUDA everything runs in csrc/kernels/delta_rule.cu (and
head_norm.cu for prompts); CPU tensors take the same arithmetic in tensor ops."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as Fn

from . import _lib
from ._lib import F, I, L, P, check, ptr, stream
from .head_norm import head_norm_gate

_lib.register_signature("xllm_delta_rule", [P] * 9 + [L, P, L] + [P] * 5 + [L, P, P, L] + [P] * 5 + [I] * 9 + [F, F, I, I, P, I, P])
_lib.register_signature("xllm_delta_chunk_bytes", [I, I, I, I], L)

_DT = {torch.bfloat16: 0, torch.float32: 1}


def round4(n):
    return (n + 3) // 4 * 4


@dataclass
class ChannelDelta:
    heads: int
    kv_heads: int                                # heads of q and k; heads / kv_heads neighbours share one
    dk: int
    dv: int
    taps: int
    q_scale: float = 1.0
    eps: float = 1e-6
    conv_w: Optional[torch.Tensor] = None        # [taps, 2 kv_heads dk + heads dv], q | k | v channels; last row: this token's
    a2: Optional[torch.Tensor] = None            # [heads dk, rank]
    dt_bias: Optional[torch.Tensor] = None       # [heads dk]
    a_log: Optional[torch.Tensor] = None         # [heads]
    norm_w: Optional[torch.Tensor] = None        # [dv]

    @property
    def channels(self):
        return 2 * self.kv_heads * self.dk + self.heads * self.dv

    def _launch(self, mode, state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out, scratch, rows, row0, blobs=None,
                max_q_len=0):
        ld = q.stride(0)
        for t in (q, k, v, r):
            assert t.stride(0) == ld and t.stride(1) == 1 and t.dtype == q.dtype
        H, dk, dv = self.heads, self.dk, self.dv
        assert state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (H, dk, round4(dv))
        assert ring.dtype == q.dtype and ring.is_contiguous() and ring.shape[1:] == (self.taps, self.channels)
        assert slots.dtype == torch.int32 and kv_lens.dtype == torch.int32 and zb.dtype == torch.float32 and zb.stride(1) == 1
        qn, kn, vn, gn, o = (*scratch, None)[:5]
        check(_lib.load().xllm_delta_rule(
            ptr(state), ptr(ring), ptr(slots), ptr(cu_q), ptr(kv_lens), ptr(q), ptr(k), ptr(v), ptr(r), ld, ptr(zb), zb.stride(0),
            ptr(self.conv_w), ptr(self.a2), ptr(self.dt_bias), ptr(self.a_log), ptr(gate), gate.stride(0), ptr(self.norm_w),
            ptr(out), out.stride(0), ptr(qn), ptr(kn), ptr(vn), ptr(gn), ptr(o), slots.shape[0], rows, row0, H, self.kv_heads,
            dk, dv, self.taps, self.a2.shape[1], self.q_scale, self.eps, _DT[q.dtype], mode, ptr(blobs), max_q_len, stream()),
            "delta_rule")
        from . import _count
        _count(3 if mode == 0 else 2 + mode + int(self.taps > 1))

    def _scratch(self, rows, device):
        """q, k, v behind the convolutions and the decays."""
        H, G, dkp, f32 = self.heads, self.kv_heads, round4(self.dk), dict(dtype=torch.float32, device=device)
        return (torch.empty((rows, G, dkp), **f32), torch.empty((rows, G, dkp), **f32), torch.empty((rows, H, round4(self.dv)), **f32),
                (torch.zeros if dkp != self.dk else torch.empty)((rows, H, dkp), **f32))

    def decode(self, state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out):
        """One token per sequence (sequence s is row s; cu_q [B + 1] counts up by one); `out` [B, heads * dv] is filled with
        finished rows.  Rows with a negative slot are padding."""
        B = slots.shape[0]
        if q.is_cuda and (self.dk > 256 or self.dv > 128):
            return self.prefill(state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out, padded=True)
        if not q.is_cuda:
            return self._cpu(state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out)
        self._launch(0, state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out, self._scratch(B, q.device), B, 0)
        return out

    def prefill(self, state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out, row0=0, padded=False,
                max_q_len=None, token_by_token=False):
        """Prompt rows of several sequences (absolute token rows cu_q, all at or behind row0); fills rows [row0, T) of `out`.
        `padded`: rows outside every sequence exist and must come out finite.  `max_q_len`: the most rows any sequence has
        (default: all rows).  `token_by_token`: the fp32 recurrence instead of the chunked form."""
        if not q.is_cuda:
            return self._cpu(state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out)
        T = q.shape[0]
        scratch = (*self._scratch(T, q.device), (torch.zeros if padded else torch.empty)((T, self.heads, self.dv),
                                                                                         dtype=torch.float32, device=q.device))
        blobs, n = None, slots.shape[0]
        if q.dtype == torch.bfloat16 and self.dk <= 256 and not token_by_token:
            blobs = torch.empty(_lib.load().xllm_delta_chunk_bytes(T, n, self.heads, self.dk), dtype=torch.uint8, device=q.device)
        self._launch(1 if blobs is None else 2, state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out, scratch, T, row0,
                     blobs, int(max_q_len or T))
        head_norm_gate(scratch[4][row0:], out[row0:], g=gate[row0:], w=self.norm_w, act="sigmoid", eps=self.eps)
        return out

    # ------------------------------------------------------------------ tensor-op form
    def _cpu(self, state, ring, slots, cu_q, kv_lens, q, k, v, r, zb, gate, out):
        H, G, dk, dv, taps = self.heads, self.kv_heads, self.dk, self.dv, self.taps
        x = torch.cat([q, k, v], dim=1)
        w = self.conv_w.float().T.contiguous()
        share = torch.arange(H) // (H // G)
        for i in range(slots.shape[0]):
            b, e, slot = int(cu_q[i]), int(cu_q[i + 1]), int(slots[i])
            if slot < 0 or e <= b:
                continue
            n, first = e - b, int(kv_lens[i]) - (e - b)
            old = [ring[slot, p % taps] if p >= 0 else torch.zeros_like(ring[slot, 0]) for p in range(first - taps + 1, first)]
            full = torch.cat([torch.stack(old), x[b:e]]) if taps > 1 else x[b:e]
            y = Fn.silu(Fn.conv1d(full.float().T[None], w[:, None], groups=w.shape[0])[0].T)
            for j in range(max(0, n - taps), n):
                ring[slot, (first + j) % taps] = x[b + j]
            qc, kc, vc = y.split([G * dk, G * dk, H * dv], dim=1)
            unit = lambda t: t / torch.sqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)
            qc = (unit(qc.reshape(n, G, dk)) * self.q_scale)[:, share]
            kc = unit(kc.reshape(n, G, dk))[:, share]
            vc = vc.reshape(n, H, dv)
            z = r[b:e].float() @ self.a2.float().T + self.dt_bias.float()
            g = torch.exp(-torch.exp(self.a_log.float())[None, :, None] * Fn.softplus(z, threshold=1e9).view(n, H, dk))
            beta = torch.sigmoid(zb[b:e, :H])
            S = state[slot, :, :, :dv].clone() if first > 0 else torch.zeros(H, dk, dv)
            o = torch.empty(n, H, dv)
            for t in range(n):
                S = g[t][:, :, None] * S
                u = beta[t][:, None] * (vc[t] - torch.einsum("hkv,hk->hv", S, kc[t]))
                S = S + kc[t][:, :, None] * u[:, None, :]
                o[t] = torch.einsum("hkv,hk->hv", S, qc[t])
            state[slot, :, :, :dv] = S
            head_norm_gate(o, out[b:e], g=gate[b:e], w=self.norm_w, act="sigmoid", eps=self.eps)
        return out
