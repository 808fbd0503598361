"""A mixer behind a short convolution: its input h becomes ``h + conv(h)``,

    conv(h)_t = sum_j taps[:, j] * h_(t - K + 1 + j)          per channel, h = 0 before a sequence's start

in float32; the mixer receives the result in the engine's type.  The last K - 1 inputs are per-request state beside
the mixer's own.  Where the mixer reads the float32 residual stream itself, the branch that waits to be added to the
stream - scaled, or first passed through an RMS norm of its own - is summed by the convolution's kernel in the same
pass (``forward_stream``): that kernel reads sums of neighbouring tokens, so the sum goes to another buffer, which is
the stream from then on.
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch

from .. import kernels
from ..config.plan import InputConvSpec
from ..weights.loader import WeightSpec
from .base import LayerCache, Mixer, StepContext, build_part, part_class, register_mixer
from .norm import RMSNorm

_CONV = "conv"          # the name of the carried inputs among the layer's state


class InputConv(Mixer):
    kind = "input_conv"
    takes_stream = True

    def __init__(self, spec: InputConvSpec, prefix: str, dtype, device):
        super().__init__(spec, prefix, dtype, device)
        if not (1 <= spec.taps <= kernels.CONV_MAX_TAPS):
            raise ValueError(f"a short convolution has 1 to {kernels.CONV_MAX_TAPS} taps, got {spec.taps}")
        self.inner: Mixer = build_part("mixer", spec.inner, prefix + spec.inner_name, dtype, device)
        self.graph_safe = bool(self.inner.graph_safe)
        self.taps = None

    @classmethod
    def weight_specs(cls, spec: InputConvSpec, prefix: str) -> List[WeightSpec]:
        return (part_class("mixer", spec.inner.kind).weight_specs(spec.inner, prefix + spec.inner_name)
                + [WeightSpec(prefix + spec.name, (spec.hidden, spec.taps), "around_zero")])

    def children(self):
        return (self.inner,)

    def load(self, store) -> None:
        self.inner.load(store)
        self.taps = store.get(self.prefix + self.spec.name, self.device, torch.float32).float().contiguous()

    def cache_need(self):
        return self.inner.cache_need()

    def state_need(self) -> Optional[Dict]:
        out = {"inner." + name: v for name, v in (self.inner.state_need() or {}).items()}
        if self.spec.taps > 1:
            out[_CONV] = ((self.spec.taps - 1, self.spec.hidden), torch.float32)
        return out or None

    def prepare_step(self, ctx: StepContext, cache: Optional[LayerCache]) -> None:
        self.inner.prepare_step(ctx, cache)

    def accepts_addend(self, addend) -> bool:
        """Whether the kernel forms this addition itself."""
        return (self.spec.taps <= kernels.STREAM_CONV_FUSED_TAPS and addend.gain is None
                and addend.t.dtype == torch.float32
                and (addend.norm is None or RMSNorm.accepts_branch_norm(addend.norm)))

    def forward_stream(self, x: torch.Tensor, addend, ctx: StepContext, cache, state=None,
                       writes_cache: bool = True) -> Tuple[torch.Tensor, torch.Tensor]:
        """(the mixer's result, the stream with ``addend`` - one ``accepts_addend`` took, or None - added)."""
        ws = ctx.workspace
        T, C = x.shape
        stream = x.dtype == torch.float32
        kw = {}
        total = x
        if not stream:          # a stream in the engine's type is widened for the convolution
            wide = ws.get("input_conv.wide", (T, C), torch.float32)
            kernels.widen_bf16(wide, x)
            x = wide
        elif addend is not None:
            total = ws.get("input_conv.sum", (T, C), torch.float32)
            if total.data_ptr() == x.data_ptr():        # the layer before left the stream here
                total = ws.get("input_conv.sum'", (T, C), torch.float32)
            norm = addend.norm
            kw = dict(branch=addend.t, branch_scale=addend.scale, sum_out=total)
            if norm is not None:
                kw.update(branch_weight=norm.weight, branch_eps=norm.spec.eps, branch_offset=norm.spec.weight_offset)
        h = ws.get("input_conv.h", (T, C), self.dtype)
        kernels.stream_conv(h, x, self.taps, (state or {}).get(_CONV), ctx.req_of_token, ctx.q_start, ctx.slots, ctx.num_entries,
                            single=ctx.all_single or ctx.fixed_shapes, **kw)
        own = {k[len("inner."):]: v for k, v in (state or {}).items() if k.startswith("inner.")} or None
        return self.inner.forward(h, ctx, cache, own, writes_cache), total

    def forward(self, x, ctx: StepContext, cache, state=None, writes_cache: bool = True):
        return self.forward_stream(x, None, ctx, cache, state, writes_cache)[0]


register_mixer("input_conv", InputConv)
