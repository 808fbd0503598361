"""Typed configuration of the Napuzen decoder, read from the keys of its own config.json, and its arrangement of
parts.

A Napuzen model lists its layers one by one (``layers``), each with its own type and sizes.  The sublayers read the
residual stream itself; the norms stand behind them, on what they return:

    x <- x + norm1(mixer(c(x)));   x <- x + norm2(ff(x))                (the second half is optional)

c(x) = x + conv(x) is a causal convolution over time, one filter per channel, beside the identity; its last inputs
are per-request state of every layer.  The mixer is one of

* ``gla``: linear attention with a matrix state per head and a decay per key channel;
* ``latent_attention``: attention over a cached latent with a rotated part, queries through a latent of their own;
* ``latent_attention_2``: attention over a cached latent without positions, within a sliding window, with a sigmoid
  gate of one number per head; such a layer may read the rows an earlier latent layer cached (``kv_from``).

The feed-forward is a gated one with a clamped swish, or a mixture of SiLU experts with a softmax router and a shared
expert behind a sigmoid gate.  The logits come from the embedding table, times ``logit_scale``.  The residual stream
is float32 whatever the engine's dtype is.

Every size and every constant that config.json gives is read here and handed to the parts through their specs; the
design fixes the tensor names, the arrangement and the constants below.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .errors import ConfigError
from .plan import (BlockOp, BlockSpec, FeedForwardSpec, GatedLinearAttentionSpec, InputConvSpec, LatentAttentionSpec,
                   LayerRun, ModelPlan, NormSpec, RopeSpec, RoutedExpertsSpec, YarnScaling)
from .reading import integer as _int, need as _get, number as _num

ARCHITECTURE = "Napuzen"
# the engine's own bound on a sequence: this design has no position table and names no limit
MAX_POSITIONS = 1 << 20
# constants of the design
SWISH_ALPHA = 1.702            # the dense feed-forward's gate: a * sigmoid(1.702 a)
WEIGHT_SUM_EPS = 1e-20         # added to the sum that the chosen experts' scores are divided by
LATENT_TYPES = ("latent_attention", "latent_attention_2")


@dataclass(frozen=True)
class NapuzenRot:
    dims: int
    base: float
    scaling: Optional[YarnScaling]


@dataclass(frozen=True)
class NapuzenMixer:
    """Sizes of a layer's mixer; those a type does not have stay at their defaults."""
    heads: int
    dim: int                      # query/key channels of a head (latent attention: the channels that are not rotated)
    vdim: int
    tau: float = 1.0              # gla
    scale: float = 1.0            # latent attention, both types
    kv_rank: int = 0
    q_rank: int = 0               # latent_attention
    rot_dim: int = 0
    rot: Optional[NapuzenRot] = None
    window: Optional[int] = None  # latent_attention_2
    kv_from: Optional[int] = None


@dataclass(frozen=True)
class NapuzenMlp:
    """``kind`` "dense": ``ff``, ``limit``.  "moe": ``ff`` of an expert, the router's ``experts``, ``top``, ``scale``
    and the width of the shared expert (None: there is none)."""
    kind: str
    ff: int
    limit: float = 0.0
    experts: int = 0
    top: int = 0
    scale: float = 1.0
    shared_ff: Optional[int] = None


@dataclass(frozen=True)
class NapuzenLayer:
    type: str
    mixer: NapuzenMixer
    mlp: Optional[NapuzenMlp]


def _rot(raw, where: str, most: int) -> NapuzenRot:
    dims = _int(raw, "dims", where, least=2)
    if dims % 2 or dims > most:
        raise ConfigError(f"'{where}dims' {dims} must be even and at most {most}")
    scaling = None
    if raw.get("scaling") is not None:
        s, ws = raw["scaling"], where + "scaling."
        scaling = YarnScaling(factor=_num(s, "factor", ws, True), original=_num(s, "original", ws, True),
                              fast=_num(s, "fast", ws, True), slow=_num(s, "slow", ws, True))
    return NapuzenRot(dims, _num(raw, "base", where, True), scaling)


def _mixer(kind: str, m, wm: str) -> NapuzenMixer:
    sizes = dict(heads=_int(m, "heads", wm), dim=_int(m, "dim", wm), vdim=_int(m, "vdim", wm))
    if kind == "gla":
        return NapuzenMixer(**sizes, tau=_num(m, "tau", wm, positive=True))
    latent = dict(scale=_num(m, "scale", wm), kv_rank=_int(m, "kv_rank", wm))
    if kind == LATENT_TYPES[0]:
        rot_dim = _int(m, "rot_dim", wm, least=2)
        return NapuzenMixer(**sizes, **latent, q_rank=_int(m, "q_rank", wm), rot_dim=rot_dim,
                            rot=_rot(_get(m, "rot", wm), wm + "rot.", rot_dim))
    kv_from = _int(m, "kv_from", wm, least=0) if m.get("kv_from") is not None else None
    return NapuzenMixer(**sizes, **latent, window=_int(_get(m, "mask", wm), "size", wm + "mask."), kv_from=kv_from)


def _mlp(f, wf: str) -> NapuzenMlp:
    kind = _get(f, "kind", wf)
    if kind == "dense":
        return NapuzenMlp("dense", ff=_int(f, "ff", wf), limit=_num(f, "limit", wf, positive=True))
    if kind != "moe":
        raise ConfigError(f"config key '{wf}kind' is '{kind}'; known: dense, moe")
    r, wr = _get(f, "router", wf), wf + "router."
    experts, top = _int(r, "experts", wr), _int(r, "top", wr)
    if top > experts:
        raise ConfigError(f"'{wr}top' {top} is more than '{wr}experts' {experts}")
    shared = _int(f["shared"], "ff", wf + "shared.") if f.get("shared") is not None else None
    return NapuzenMlp("moe", ff=_int(_get(f, "expert", wf), "ff", wf + "expert."), experts=experts, top=top,
                      scale=_num(r, "scale", wr), shared_ff=shared)


@dataclass(frozen=True)
class NapuzenConfig:
    vocab: int
    width: int
    eps: float
    conv_taps: int
    logit_scale: float
    layers: Tuple[NapuzenLayer, ...]

    ARCHITECTURE = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "NapuzenConfig":
        vocab, width = _int(raw, "vocab", ""), _int(raw, "width", "")
        eps = _num(_get(raw, "norm", ""), "eps", "norm.", positive=True)
        taps = _int(_get(raw, "canon", ""), "taps", "canon.")
        logit_scale = _num(raw, "logit_scale", "")
        layers = _get(raw, "layers", "")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config key 'layers' must be a non-empty list")
        out = []
        for i, layer in enumerate(layers):
            w = f"layers[{i}]."
            kind = _get(layer, "type", w)
            if kind != "gla" and kind not in LATENT_TYPES:
                raise ConfigError(f"config key '{w}type' is '{kind}'; known: gla, {', '.join(LATENT_TYPES)}")
            mixer = _mixer(kind, _get(layer, "mixer", w), w + "mixer.")
            mlp = _mlp(layer["mlp"], w + "mlp.") if layer.get("mlp") is not None else None
            out.append(NapuzenLayer(kind, mixer, mlp))
        for i, layer in enumerate(out):
            j = layer.mixer.kv_from
            if j is None:
                continue
            if not (0 <= j < i) or out[j].type not in LATENT_TYPES or out[j].mixer.kv_from is not None:
                raise ConfigError(f"'layers[{i}].mixer.kv_from' {j} must name an earlier latent attention layer with a latent "
                                  f"projection of its own")
            if layer.mixer.kv_rank != out[j].mixer.kv_rank:
                raise ConfigError(f"layer {i} reads the cached rows of layer {j}: their kv_rank must be equal")
        return cls(vocab=vocab, width=width, eps=eps, conv_taps=taps, logit_scale=logit_scale, layers=tuple(out))

    # ---- the arrangement of parts ---------------------------------------------------------
    def _latent_spec(self, i: int, keep) -> LatentAttentionSpec:
        m = self.layers[i].mixer
        owner = i if m.kv_from is None else m.kv_from
        common = dict(kind="latent_attention", hidden=self.width, num_heads=m.heads, head_dim=m.dim, v_head_dim=m.vdim,
                      kv_rank=m.kv_rank, scale=m.scale, norm_eps=self.eps, window=m.window, cache_window=keep[owner])
        if self.layers[i].type == "latent_attention":
            # the rotary magnitude: cos and sin grow with the logarithm of the stretch
            magnitude = 0.1 * math.log(m.rot.scaling.factor) + 1.0 if m.rot.scaling is not None else 1.0
            rope = RopeSpec(kind="rope", head_dim=m.rot_dim, rotary_dim=m.rot.dims, theta=m.rot.base,
                            max_positions=MAX_POSITIONS, layout="interleaved", scaling=m.rot.scaling, tables=False,
                            magnitude=magnitude)
            return LatentAttentionSpec(**common, rope_dim=m.rot_dim, rope=rope, q_rank=m.q_rank)
        return LatentAttentionSpec(**common, gate=True, gate_per_head=True, shares_cache=m.kv_from is not None,
                                   row_tail=self.layers[owner].mixer.rot_dim)

    def plan(self) -> ModelPlan:
        def norm():
            return NormSpec(kind="rmsnorm", dim=self.width, eps=self.eps, weight_offset=0.0, weight_name="")

        def gated(ff: int, activation: str, params=()):
            return FeedForwardSpec(kind="swiglu", hidden=self.width, intermediate=ff, activation=activation,
                                   names=("gate", "up", "down"), act_params=tuple(params))

        # rows cached by a latent layer are kept as long as the widest window among its readers asks
        windows = {}
        for i, layer in enumerate(self.layers):
            if layer.type in LATENT_TYPES:
                m = layer.mixer
                windows.setdefault(i if m.kv_from is None else m.kv_from, []).append(m.window)
        keep = {j: None if any(w is None for w in ws) else max(ws) for j, ws in windows.items()}

        blocks, runs = [], []
        for i, layer in enumerate(self.layers):
            m = layer.mixer
            if layer.type == "gla":
                inner = GatedLinearAttentionSpec(kind="gated_linear_attention", hidden=self.width, heads=m.heads,
                                                 head_dim=m.dim, v_head_dim=m.vdim, tau=m.tau, eps=self.eps)
            else:
                inner = self._latent_spec(i, keep)
            mixer = InputConvSpec(kind="input_conv", hidden=self.width, inner=inner, taps=self.conv_taps, name="canon1",
                                  inner_name="mix.")
            prog = [BlockOp("mixer", "x", "a", mixer),
                    BlockOp("norm", "a", "a", norm(), "norm1"),
                    BlockOp("add", "a", "x")]
            if layer.mlp is not None:
                f = layer.mlp
                if f.kind == "dense":
                    ff = gated(f.ff, "swish_clamp", (f.limit, SWISH_ALPHA))
                else:
                    ff = RoutedExpertsSpec(kind="routed_experts", hidden=self.width, intermediate=f.ff, experts=f.experts,
                                           top=f.top, correction=False, score="softmax", renormalize=True,
                                           renormalize_eps=WEIGHT_SUM_EPS, weight_scale=f.scale, activation="silu",
                                           shared=gated(f.shared_ff, "silu") if f.shared_ff is not None else None,
                                           shared_gate="shared.sg" if f.shared_ff is not None else None)
                # the feed-forward reads the stream itself: its "norm" hands the sum over in the engine's type
                prog += [BlockOp("norm", "x", "h", NormSpec(kind="identity", dim=self.width), "stream"),
                         BlockOp("feed_forward", "h", "f", ff, "mlp."),
                         BlockOp("norm", "f", "f", norm(), "norm2"),
                         BlockOp("add", "f", "x")]
            blocks.append(BlockSpec(f"l{i}.", tuple(prog)))
            runs.append(LayerRun(block=i, cache_from=m.kv_from))
        plan = ModelPlan(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden=self.width, embed_name="embed",
            blocks=tuple(blocks), runs=tuple(runs), final_norm=norm(), final_norm_name="final.norm", head_name=None,
            max_positions=MAX_POSITIONS, logit_scale=self.logit_scale, residual_dtype="float32")
        plan.validate()
        return plan
