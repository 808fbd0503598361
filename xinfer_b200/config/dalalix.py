"""Typed configuration of the Dalalix decoder, read from the keys of its own config.json, and its arrangement of
parts.

A Dalalix model lists its layers one by one (``layers``), each with its own type and sizes.  There is no single residual
stream but ``streams`` of them, all equal to the embedding's output at first.  Half a layer (mixer or feed-forward) reads
one weighted sum of them and writes to all:

    u = sum_s r[s] X[s];   y = sublayer(norm(u));   X[t] <- sum_s M[s, t] X[s] + w[t] y        (the second half is optional)

The final norm reads the streams' plain sum.  A token's embedding row gets a row of a hashed (token before, token) table
added.  The mixer is one of

* ``attention``: grouped-query attention without positions; q, k and v pass a short causal convolution, values are
  divided by their root mean square, the heads' outputs are gated per channel;
* ``attention_2``: grouped-query attention without positions, with biases on q, k and v;
* ``parallel``: attention with biases, rotation, a sliding window that keeps a sequence's first tokens and a learned
  sink per head, beside a matrix memory with exponential gates.

The feed-forward is a mixture of clamped swish experts with a softmax router that chooses among groups.  A layer may
use another layer's weights (``weights_of``) with a cache and state of its own.

Every size and every constant that config.json gives is read here and handed to the parts through their specs; the
design fixes the tensor names, the arrangement and the constants below.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .errors import ConfigError
from .plan import (AttentionSpec, BlockOp, BlockSpec, LayerRun, MatrixMemorySpec, ModelPlan, NormSpec, PairEmbeddingSpec,
                   ParallelMixerSpec, RopeSpec, RoutedExpertsSpec, StreamMixSpec)
from .reading import integer as _int, need as _get, number as _num

ARCHITECTURE = "Dalalix"
# the engine's own bound on a sequence: this design has no position table and names no limit
MAX_POSITIONS = 1 << 20
# constants of the design
SWISH_ALPHA = 1.702            # an expert's gate: a * sigmoid(1.702 a)
WEIGHT_SUM_EPS = 1e-20         # added to the sum that the chosen experts' scores are divided by
GROUP_BEST = 1                 # a group of experts is as good as its best one
MEMORY_DIVISOR_EPS = 1e-6      # beside the matrix memory's divisor


@dataclass(frozen=True)
class DalalixAttention:
    """Sizes of a softmax attention; what a type does not have stays at its default.  ``rot`` = (dims, base)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: Optional[int] = None
    rot: Optional[Tuple[int, float]] = None
    window: Optional[int] = None
    keep_first: int = 0


@dataclass(frozen=True)
class DalalixMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class DalalixParallel:
    left: DalalixAttention
    right: DalalixMemory
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class DalalixMlp:
    ff: int
    limit: float
    experts: int
    top: int
    groups: int
    keep: int


@dataclass(frozen=True)
class DalalixLayer:
    type: str
    mixer: Union[DalalixAttention, DalalixParallel]
    mlp: Optional[DalalixMlp]
    weights_of: Optional[int] = None


def _attention(m, wm: str, **more) -> DalalixAttention:
    heads, kv = _int(m, "heads", wm), _int(m, "kv_heads", wm)
    if heads % kv:
        raise ConfigError(f"'{wm}heads' {heads} is not a multiple of '{wm}kv_heads' {kv}")
    return DalalixAttention(heads, kv, _int(m, "dim", wm), _int(m, "vdim", wm), _num(m, "scale", wm), **more)


def _mixer(kind: str, m, wm: str):
    if kind == "attention":
        return _attention(m, wm, conv=_int(m, "conv", wm))
    if kind == "attention_2":
        return _attention(m, wm)
    left, wl = _get(m, "left", wm), wm + "left."
    right, wr = _get(m, "right", wm), wm + "right."
    rot = None
    if left.get("rot") is not None:
        r, wrot = left["rot"], wl + "rot."
        dims = _int(r, "dims", wrot, least=0)
        if dims % 2 or dims > _int(left, "dim", wl):
            raise ConfigError(f"'{wrot}dims' {dims} must be even and at most '{wl}dim' {left['dim']}")
        if dims:
            rot = (dims, _num(r, "base", wrot, positive=True))
    mask, wmask = _get(left, "mask", wl), wl + "mask."
    return DalalixParallel(
        left=_attention(left, wl, rot=rot, window=_int(mask, "size", wmask), keep_first=_int(mask, "keep_first", wmask, least=0)),
        right=DalalixMemory(_int(right, "heads", wr), _int(right, "dim", wr), _int(right, "vdim", wr),
                            _num(right, "gate_cap", wr, positive=True)),
        left_scale=_num(m, "left_scale", wm), right_scale=_num(m, "right_scale", wm))


def _mlp(f, wf: str) -> DalalixMlp:
    kind = _get(f, "kind", wf)
    if kind != "moe":
        raise ConfigError(f"config key '{wf}kind' is '{kind}'; known: moe")
    e, we = _get(f, "expert", wf), wf + "expert."
    r, wr = _get(f, "router", wf), wf + "router."
    experts, top = _int(r, "experts", wr), _int(r, "top", wr)
    groups, keep = 1, 1
    if r.get("groups") is not None:
        groups, keep = _int(r["groups"], "count", wr + "groups."), _int(r["groups"], "keep", wr + "groups.")
    if experts % groups or keep > groups:
        raise ConfigError(f"'{wr}experts' {experts} do not form {groups} equal groups of which {keep} are kept")
    if top > keep * (experts // groups):
        raise ConfigError(f"'{wr}top' {top} is more than the {keep} kept groups of {experts // groups} experts hold")
    return DalalixMlp(_int(e, "ff", we), _num(e, "limit", we, positive=True), experts, top, groups, keep)


LAYER_TYPES = ("attention", "attention_2", "parallel")


@dataclass(frozen=True)
class DalalixConfig:
    vocab: int
    width: int
    eps: float
    streams: int
    bigram: Optional[Tuple[int, int, int]]      # buckets, mul_prev, mul_cur
    logit_softcap: Optional[float]
    layers: Tuple[DalalixLayer, ...]

    ARCHITECTURE = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "DalalixConfig":
        vocab, width = _int(raw, "vocab", ""), _int(raw, "width", "")
        eps = _num(_get(raw, "norm", ""), "eps", "norm.", positive=True)
        streams = _int(raw, "streams", "")
        softcap = _num(raw, "logit_softcap", "", positive=True) if raw.get("logit_softcap") is not None else None
        bigram = None
        emb = raw.get("embedding") or {}
        if emb.get("bigram") is not None:
            b, wb = emb["bigram"], "embedding.bigram."
            bigram = (_int(b, "buckets", wb), _int(b, "mul_prev", wb, least=0), _int(b, "mul_cur", wb, least=0))
        layers = _get(raw, "layers", "")
        if not isinstance(layers, (list, tuple)) or not layers:
            raise ConfigError("config key 'layers' must be a non-empty list")
        out = []
        for i, layer in enumerate(layers):
            w = f"layers[{i}]."
            kind = _get(layer, "type", w)
            if kind not in LAYER_TYPES:
                raise ConfigError(f"config key '{w}type' is '{kind}'; known: {', '.join(LAYER_TYPES)}")
            mixer = _mixer(kind, _get(layer, "mixer", w), w + "mixer.")
            mlp = _mlp(layer["mlp"], w + "mlp.") if layer.get("mlp") is not None else None
            of = _int(layer, "weights_of", w, least=0) if layer.get("weights_of") is not None else None
            out.append(DalalixLayer(kind, mixer, mlp, of))
        for i, layer in enumerate(out):
            j = layer.weights_of
            if j is None:
                continue
            if j >= len(out) or j == i or out[j].weights_of is not None:
                raise ConfigError(f"'layers[{i}].weights_of' {j} must name a layer with weights of its own")
            if (layer.type, layer.mixer, layer.mlp) != (out[j].type, out[j].mixer, out[j].mlp):
                raise ConfigError(f"layer {i} uses the weights of layer {j}, but the two differ in type or sizes")
        return cls(vocab=vocab, width=width, eps=eps, streams=streams, bigram=bigram, logit_softcap=softcap, layers=tuple(out))

    # ---- the arrangement of parts ---------------------------------------------------------
    def _attention_spec(self, m: DalalixAttention, **more) -> AttentionSpec:
        rope = None
        if m.rot is not None:
            rope = RopeSpec(kind="rope", head_dim=m.dim, rotary_dim=m.rot[0], theta=m.rot[1], max_positions=MAX_POSITIONS,
                            layout="neox", tables=False)
        return AttentionSpec(kind="talking_attention", hidden=self.width, num_heads=m.heads, num_kv_heads=m.kv_heads,
                             head_dim=m.dim, v_head_dim=m.vdim, scale=m.scale, rope=rope, window=m.window,
                             keep_first=m.keep_first, names=("q", "k", "v", "o", "talk"), **more)

    def _mixer_spec(self, layer: DalalixLayer):
        m = layer.mixer
        if layer.type == "attention":
            return self._attention_spec(m, conv=m.conv, value_norm_eps=self.eps, gate_name="g")
        if layer.type == "attention_2":
            return self._attention_spec(m, bias_suffix=".b")
        memory = MatrixMemorySpec(kind="matrix_memory", hidden=self.width, heads=m.right.heads, head_dim=m.right.dim,
                                  v_head_dim=m.right.vdim, gate_cap=m.right.gate_cap, eps=self.eps,
                                  divisor_eps=MEMORY_DIVISOR_EPS)
        return ParallelMixerSpec(kind="parallel", hidden=self.width,
                                 left=self._attention_spec(m.left, bias_suffix=".b", sink_name="sink"), right=memory,
                                 left_scale=m.left_scale, right_scale=m.right_scale)

    def plan(self) -> ModelPlan:
        def norm():
            return NormSpec(kind="rmsnorm", dim=self.width, eps=self.eps, weight_offset=0.0, weight_name="")

        def mix(q: int):
            return StreamMixSpec(self.streams, (f"hc{q}.in", f"hc{q}.mix", f"hc{q}.out"))

        blocks, block_of = [], {}
        for i, layer in enumerate(self.layers):
            if layer.weights_of is not None:
                continue
            prog = [BlockOp("norm", "x", "h", norm(), "norm1", mix=mix(1)),
                    BlockOp("mixer", "h", "a", self._mixer_spec(layer), "mix."),
                    BlockOp("add", "a", "x", mix=mix(1))]
            if layer.mlp is not None:
                f = layer.mlp
                ff = RoutedExpertsSpec(kind="routed_experts", hidden=self.width, intermediate=f.ff, experts=f.experts,
                                       top=f.top, groups=f.groups, keep=f.keep, group_best=GROUP_BEST, correction=False,
                                       score="softmax", renormalize=True, renormalize_eps=WEIGHT_SUM_EPS,
                                       activation="swish_clamp", act_params=(f.limit, SWISH_ALPHA))
                prog += [BlockOp("norm", "x", "h", norm(), "norm2", mix=mix(2)),
                         BlockOp("feed_forward", "h", "f", ff, "mlp."),
                         BlockOp("add", "f", "x", mix=mix(2))]
            block_of[i] = len(blocks)
            blocks.append(BlockSpec(f"l{i}.", tuple(prog)))
        runs = tuple(LayerRun(block=block_of[i if layer.weights_of is None else layer.weights_of])
                     for i, layer in enumerate(self.layers))
        pair = PairEmbeddingSpec("bigram", *self.bigram) if self.bigram is not None else None
        plan = ModelPlan(
            architecture=ARCHITECTURE, vocab_size=self.vocab, hidden=self.width, embed_name="embed",
            blocks=tuple(blocks), runs=runs, final_norm=norm(), final_norm_name="final.norm", head_name="head",
            max_positions=MAX_POSITIONS, logit_softcap=self.logit_softcap, residual_dtype="float32", pair_embedding=pair,
            streams=self.streams)
        plan.validate()
        return plan
