"""Matrix memory with exponential gates and a running maximum (mLSTM):

    m' = max(f + m, i);  S <- e^(f + m - m') S + e^(i - m') k v^T;  n likewise with k;  o = S^T q / (max(|n.q|, e^-m') + 1e-6)

`MatrixMemory` carries the constants of one layer; its methods take column blocks of the layer's projection rows as they
are, and fp32 gate projections.  On CUDA everything runs in csrc/kernels/mlstm.cu (and head_norm.cu for prompts); CPU
tensors take the same arithmetic in tensor ops."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _lib
from ._lib import F, I, L, P, check, ptr, stream
from .delta_rule import round4
from .head_norm import head_norm_gate

_lib.register_signature("xllm_mlstm", [P] * 9 + [L, P, P, L, P, L, P, P, L, P, P, P] + [I] * 5 + [F] * 3 + [I, I, P])

_DT = {torch.bfloat16: 0, torch.float32: 1}


@dataclass
class MatrixMemory:
    heads: int
    dk: int
    dv: int
    cap: float                                   # of both gates: cap tanh(z / cap)
    q_scale: float = 1.0
    eps: float = 1e-6
    norm_w: Optional[torch.Tensor] = None        # [heads * dv]

    def _launch(self, mode, st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out, o, div, gates=None):
        ld = q.stride(0)
        for t in (q, k, v):
            assert t.stride(0) == ld and t.stride(1) == 1 and t.dtype == q.dtype
        S, n, m = st["S"], st["n"], st["m"]
        H, dk, dv = self.heads, self.dk, self.dv
        assert S.shape[1:] == (H, dk, round4(dv)) and n.shape[1:] == (H, dk) and m.shape[1:] == (H,)
        assert all(t.dtype == torch.float32 and t.is_contiguous() for t in (S, n, m))
        assert zi.dtype == zf.dtype == torch.float32 and zi.stride() == zf.stride() and zi.stride(1) == 1
        assert slots.dtype == torch.int32 and kv_lens.dtype == torch.int32
        check(_lib.load().xllm_mlstm(
            ptr(S), ptr(n), ptr(m), ptr(slots), ptr(cu_q), ptr(kv_lens), ptr(q), ptr(k), ptr(v), ld, ptr(zi), ptr(zf),
            zi.stride(0), ptr(gate), gate.stride(0), ptr(self.norm_w), ptr(out), out.stride(0), ptr(o), ptr(div),
            ptr(gates), q.shape[0], slots.shape[0], H, dk, dv, self.q_scale, self.cap, self.eps, _DT[q.dtype], mode, stream()), "mlstm")
        from . import _count
        _count(1 if mode == 0 else 2)

    def decode(self, st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out):
        """One token per sequence (sequence s is row s; cu_q [B + 1] counts up by one); `out` [B, heads * dv] is filled with
        finished rows.  st: the layer's state tensors S, n, m.  Rows with a negative slot are padding."""
        if q.is_cuda and (self.dk > 256 or self.dv > 128):
            return self.prefill(st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out, padded=True)
        if not q.is_cuda:
            return self._cpu(st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out)
        self._launch(0, st, slots, None, kv_lens, q, k, v, zi, zf, gate, out, None, None)
        return out

    def prefill(self, st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out, row0=0, padded=False,
                token_by_token=False):
        """Prompt rows of several sequences (absolute token rows cu_q, all at or behind row0); fills rows [row0, T) of `out`.
        `padded`: rows outside every sequence exist and must come out finite.  `token_by_token`: the fp32 recurrence instead of
        the chunked form."""
        if not q.is_cuda:
            return self._cpu(st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out)
        make = torch.zeros if padded else torch.empty
        o = make((q.shape[0], self.heads, self.dv), dtype=torch.float32, device=q.device)
        div = make((q.shape[0], self.heads), dtype=torch.float32, device=q.device)
        gates = None
        if q.dtype == torch.bfloat16 and not token_by_token:
            T, n = q.shape[0], slots.shape[0]
            gates = torch.empty(self.heads * (3 * T + T // 16 + n + 1), dtype=torch.float32, device=q.device)
        self._launch(1 if gates is None else 2, st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out, o, div, gates)
        head_norm_gate(o[row0:], out[row0:], div=div[row0:], g=gate[row0:], w=self.norm_w, act="sigmoid", eps=self.eps)
        return out

    # ------------------------------------------------------------------ tensor-op form
    def _cpu(self, st, slots, cu_q, kv_lens, q, k, v, zi, zf, gate, out):
        H, dk, dv, cap = self.heads, self.dk, self.dv, self.cap
        for i in range(slots.shape[0]):
            b, e, slot = int(cu_q[i]), int(cu_q[i + 1]), int(slots[i])
            if slot < 0 or e <= b:
                continue
            n = e - b
            qf = q[b:e].float().reshape(n, H, dk) * self.q_scale
            kf, vf = k[b:e].float().reshape(n, H, dk), v[b:e].float().reshape(n, H, dv)
            il = cap * torch.tanh(zi[b:e] / cap)
            fl = torch.nn.functional.logsigmoid(cap * torch.tanh(zf[b:e] / cap))
            if int(kv_lens[i]) == n:
                S, N, m = torch.zeros(H, dk, dv), torch.zeros(H, dk), torch.zeros(H)
            else:
                S, N, m = st["S"][slot, :, :, :dv].clone(), st["n"][slot].clone(), st["m"][slot].clone()
            o, div = torch.empty(n, H, dv), torch.empty(n, H)
            for t in range(n):
                new = torch.maximum(fl[t] + m, il[t])
                keep, write = torch.exp(fl[t] + m - new), torch.exp(il[t] - new)
                m = new
                kw = kf[t] * write[:, None]
                S = keep[:, None, None] * S + kw[:, :, None] * vf[t][:, None, :]
                N = keep[:, None] * N + kw
                o[t] = torch.einsum("hkv,hk->hv", S, qf[t])
                div[t] = torch.maximum((N * qf[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
            st["S"][slot, :, :, :dv], st["n"][slot], st["m"][slot] = S, N, m
            head_norm_gate(o, out[b:e], div=div, g=gate[b:e], w=self.norm_w, act="sigmoid", eps=self.eps)
        return out
