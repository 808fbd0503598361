"""A matrix memory per head with exponential gates, kept in range by a running maximum (xLSTM's mLSTM).

    q = W_q h head_dim^-1/2, k = W_k h (heads x head_dim), v = W_v h (heads x v_head_dim)
    i = cap tanh((W_i h + b_i) / cap),  f = logsigmoid(cap tanh((W_f h + b_f) / cap))        logarithms, per head
    m' = max(f + m, i);   S <- e^(f + m - m') S + e^(i - m') k v^T;   n <- e^(f + m - m') n + e^(i - m') k
    o  = S^T q / (max(|n . q|, e^(-m')) + divisor_eps)                the read sees the token's own write
    out = W_o ( o / rms(o) * w * sigmoid(W_g h) )                     norm per head, w over all heads' channels

ONE product [q | k | v | gate | i | f] leaves float32; the gates, the maximum, the state, its reads, the division, the
norm and the output gate are float32 in both engine types.  The scan leaves the reads and their divisors apart; the norm's
kernel divides.  A request keeps S, n and m in its row of the engine's per-request state tables (m in two places, see
csrc/state_scan.cu).
"""
from __future__ import annotations

from typing import List

import torch

from .. import kernels
from ..config.plan import MatrixMemorySpec
from ..weights.loader import WeightSpec
from .base import Mixer, StepContext, register_mixer
from .linear import linear, stack_rows


class MatrixMemory(Mixer):
    kind = "matrix_memory"
    graph_safe = True

    def __init__(self, spec: MatrixMemorySpec, prefix: str, dtype, device):
        super().__init__(spec, prefix, dtype, device)
        self.qk = spec.heads * spec.head_dim
        self.vw = spec.heads * spec.v_head_dim
        self.w_in = self.w_o = self.norm_w = self.b_in = self.b_forget = None

    @classmethod
    def weight_specs(cls, spec: MatrixMemorySpec, prefix: str) -> List[WeightSpec]:
        n, W, H = spec.names, spec.hidden, spec.heads
        qk, vw = H * spec.head_dim, H * spec.v_head_dim
        return [WeightSpec(prefix + n[0], (qk, W)), WeightSpec(prefix + n[1], (qk, W)), WeightSpec(prefix + n[2], (vw, W)),
                WeightSpec(prefix + n[3], (vw, W)), WeightSpec(prefix + n[4], (W, vw)), WeightSpec(prefix + n[5], (vw,), "norm"),
                WeightSpec(prefix + n[6], (H, W)), WeightSpec(prefix + n[7], (H,), "unit"),
                WeightSpec(prefix + n[8], (H, W)), WeightSpec(prefix + n[9], (H,), "unit")]

    def load(self, store) -> None:
        p, n = self.prefix, self.spec.names

        def operand(name):
            return store.get(p + name, self.device, self.dtype, operand=True)

        def f32(name):
            return store.get(p + name, self.device, torch.float32).float().contiguous()
        self.w_in = stack_rows([operand(n[i]) for i in (0, 1, 2, 3, 6, 8)])
        self.w_o = operand(n[4])
        self.norm_w, self.b_in, self.b_forget = f32(n[5]), f32(n[7]), f32(n[9])

    def state_need(self):
        s = self.spec
        return {"S": ((s.heads, s.head_dim, s.v_head_dim), torch.float32), "n": ((s.heads, s.head_dim), torch.float32),
                "m": ((s.heads, 2, 2), torch.float32)}

    # ---- the two halves ---------------------------------------------------------------------------
    def inner_width(self) -> int:
        return self.vw

    def output_weight(self) -> torch.Tensor:
        return self.w_o

    def forward_inner(self, x, ctx: StepContext, cache, state, writes_cache, out, out_scale) -> None:
        s = self.spec
        T, H, d, dv = x.shape[0], s.heads, s.head_dim, s.v_head_dim
        ws = ctx.workspace
        proj = ws.get("memory.proj", (T, self.w_in.shape[0]), torch.float32)
        linear(proj, x, self.w_in, ctx.err)
        o = ws.get("memory.o", (T, self.vw), torch.float32)
        div = ws.get("memory.div", (T, H), torch.float32)
        kernels.matrix_memory(o, div, proj, 2 * self.qk + 2 * self.vw, self.b_in, self.b_forget, s.gate_cap, state, ctx.q_start,
                              ctx.start_pos, ctx.slots, ctx.num_entries, H, d, dv, d ** -0.5, s.divisor_eps)
        kernels.gated_head_norm(out, o, proj, 2 * self.qk + self.vw, self.norm_w, dv, s.eps, gate_after=True, div=div,
                                out_scale=out_scale)

    def forward(self, x, ctx: StepContext, cache=None, state=None, writes_cache: bool = True):
        T = x.shape[0]
        inner = ctx.workspace.get("memory.inner", (T, self.vw), self.dtype)
        self.forward_inner(x, ctx, cache, state, writes_cache, inner, 1.0)
        out = ctx.workspace.get("memory.out", (T, self.spec.hidden), ctx.branch_dtype or self.dtype)
        linear(out, inner, self.w_o, ctx.err)
        return out


register_mixer("matrix_memory", MatrixMemory)
