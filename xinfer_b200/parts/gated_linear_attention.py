"""Linear attention with a matrix state per head that forgets per key channel.

    q = W_q h, k = W_k h (heads x head_dim), v = W_v h (heads x v_head_dim)
    alpha = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)               per head and key channel
    S <- diag(alpha) S + k v^T;  o = S^T q head_dim^-1/2       the read sees the token's own write
    out = W_o ( o / rms(o) * w * silu(W_g h) )                 norm per head, w shared by the heads

ONE product [q | k | v | gate | W_a1 h] leaves float32; the second half of the low-rank map, the decay, the state, its
reads, the norm and the gate are float32 in both engine types.  A request keeps the state matrices in its row of the
engine's per-request state tables.
"""
from __future__ import annotations

from typing import List

import torch

from .. import kernels
from ..config.plan import GatedLinearAttentionSpec
from ..weights.loader import WeightSpec
from .base import Mixer, StepContext, register_mixer
from .linear import linear, stack_rows


class GatedLinearAttention(Mixer):
    kind = "gated_linear_attention"
    graph_safe = True

    def __init__(self, spec: GatedLinearAttentionSpec, prefix: str, dtype, device):
        super().__init__(spec, prefix, dtype, device)
        self.qk = spec.heads * spec.head_dim
        self.vw = spec.heads * spec.v_head_dim
        self.w_in = self.w_o = self.w_decay = self.decay_bias = self.norm_w = None

    @classmethod
    def weight_specs(cls, spec: GatedLinearAttentionSpec, prefix: str) -> List[WeightSpec]:
        n, W = spec.names, spec.hidden
        qk, vw = spec.heads * spec.head_dim, spec.heads * spec.v_head_dim
        r = -1 if spec.decay_rank is None else spec.decay_rank
        R = spec.DEFAULT_RANK
        return [WeightSpec(prefix + n[0], (qk, W)), WeightSpec(prefix + n[1], (qk, W)), WeightSpec(prefix + n[2], (vw, W)),
                WeightSpec(prefix + n[3], (vw, W)), WeightSpec(prefix + n[4], (W, vw)),
                WeightSpec(prefix + n[5], (spec.v_head_dim,), "norm"),
                WeightSpec(prefix + n[6], (r, W), "linear", R), WeightSpec(prefix + n[7], (qk, r), "linear", R),
                WeightSpec(prefix + n[8], (qk,), "unit")]

    def load(self, store) -> None:
        p, n = self.prefix, self.spec.names

        def operand(name):
            return store.get(p + name, self.device, self.dtype, operand=True)

        def f32(name):
            return store.get(p + name, self.device, torch.float32).float().contiguous()
        a1 = operand(n[6])
        self.w_decay, self.decay_bias, self.norm_w = f32(n[7]), f32(n[8]), f32(n[5])
        if self.w_decay.shape[1] != a1.shape[0]:
            raise ValueError(f"'{p}': the two halves of the low-rank map disagree about its inner size")
        self.w_in = stack_rows([operand(n[0]), operand(n[1]), operand(n[2]), operand(n[3]), a1])
        self.w_o = operand(n[4])

    def state_need(self):
        s = self.spec
        return {"S": ((s.heads, s.head_dim, s.v_head_dim), torch.float32)}

    def forward(self, x, ctx: StepContext, cache=None, state=None, writes_cache: bool = True):
        s = self.spec
        T, H, d, dv = x.shape[0], s.heads, s.head_dim, s.v_head_dim
        ws = ctx.workspace
        proj = ws.get("gla.proj", (T, self.w_in.shape[0]), torch.float32)
        linear(proj, x, self.w_in, ctx.err)
        at = 2 * self.qk + 2 * self.vw
        alpha = ws.get("gla.alpha", (T, self.qk), torch.float32)
        kernels.low_rank_decay(alpha, proj[:, at:at + self.w_decay.shape[1]], self.w_decay, self.decay_bias, s.tau)
        o = ws.get("gla.o", (T, self.vw), torch.float32)
        kernels.linear_scan(o, proj, alpha, state["S"], ctx.q_start, ctx.slots, ctx.num_entries, H, d, dv, d ** -0.5)
        gated = ws.get("gla.gated", (T, self.vw), self.dtype)
        kernels.gated_head_norm(gated, o, proj, 2 * self.qk + self.vw, self.norm_w, dv, s.eps, gate_after=True, silu_gate=True)
        out = ws.get("gla.out", (T, s.hidden), ctx.branch_dtype or self.dtype)
        linear(out, gated, self.w_o, ctx.err)
        return out


register_mixer("gated_linear_attention", GatedLinearAttention)
