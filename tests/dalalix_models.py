"""Tiny Dalalix configurations for the tests (config.json dictionaries) and their random model folders.

They differ from each other in every size and switch: one to five and nine residual streams; heads, key and value sizes that
differ, that are one, that are no multiple of 16 or of 4, query groups of one to six heads; convolutions of one tap (no
state) to six; windows of one token, shorter and longer than a page and than a tile of keys, that keep no token, fewer than a
page's, and more than a tile's; rotations of none, some and all of a head; matrix memories with as many heads as the
attention beside them or not, with more or fewer value channels than key channels, with tight and wide gate caps; scales of
the two sides that are one, negative and large; routers over one to twelve experts with one to six groups that keep one, some
or all of them; layers without a feed-forward; layers that use another layer's weights once, twice and not at all, also an
earlier layer that uses a later one's; a width that is no multiple of 8; a pair table and a soft cap, or neither; vocabulary
and page size."""
from typing import Dict, List, Sequence

import numpy as np
import torch


def _soft(heads, kv, dim, vdim, scale, **more):
    return dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, **more)


def _conv(heads, kv, dim, vdim, scale, taps):
    return dict(type="attention", mixer=_soft(heads, kv, dim, vdim, scale, conv=taps), mlp=None)


def _biased(heads, kv, dim, vdim, scale):
    return dict(type="attention_2", mixer=_soft(heads, kv, dim, vdim, scale), mlp=None)


def _parallel(left, window, keep, rot, right, cap, scales):
    m = dict(_soft(*left), mask=dict(size=window, keep_first=keep))
    if rot is not None:
        m["rot"] = dict(dims=rot[0], base=rot[1])
    h, d, dv = right
    return dict(type="parallel", mlp=None, mixer=dict(left=m, right=dict(heads=h, dim=d, vdim=dv, gate_cap=cap),
                                                      left_scale=scales[0], right_scale=scales[1]))


def _moe(layer, ff, limit, experts, top, groups=None):
    router = dict(experts=experts, top=top)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(layer, mlp=dict(kind="moe", expert=dict(ff=ff, limit=limit), router=router))


def _again(layers, j):
    return dict(layers[j], weights_of=j)


def _cfg(vocab, width, eps, streams, layers, bigram=None, softcap=None):
    cfg = dict(architecture="Dalalix", vocab=vocab, width=width, norm=dict(eps=eps), streams=streams, layers=layers)
    if bigram is not None:
        cfg["embedding"] = dict(bigram=dict(buckets=bigram[0], mul_prev=bigram[1], mul_cur=bigram[2]))
    if softcap is not None:
        cfg["logit_softcap"] = softcap
    return cfg


# sizes that fit no fast path, a window shorter than a page that keeps a few tokens, three streams, weights used again
_A = [_moe(_conv(3, 1, 10, 14, 0.7, 3), 20, 0.9, 6, 2, (3, 2)),
      _moe(_parallel((4, 2, 14, 9, 0.5), 11, 5, (6, 40.0), (3, 7, 5), 4.0, (0.8, 1.3)), 24, 2.0, 5, 3),
      _biased(5, 5, 7, 12, 0.6)]
_A += [_again(_A, 1), _again(_A, 0), _again(_A, 1)]
# sizes of the tensor-core kernels: key and value heads of one size and of two, a kept range beyond a tile, more taps
_B = [_moe(_parallel((4, 2, 32, 32, 0.25), 50, 70, (32, 3000.0), (4, 32, 16), 15.0, (1.0, 1.0)), 32, 1.2, 12, 4, (4, 3)),
      _moe(_conv(6, 1, 64, 32, 0.15, 6), 40, 7.0, 8, 1, (2, 1)),
      _moe(_biased(8, 4, 16, 80, 0.4), 48, 0.6, 12, 6, (6, 5)),
      _parallel((2, 1, 128, 128, 0.11), 130, 20, (16, 1e5), (2, 48, 64), 9.0, (-0.7, 2.5))]
_B += [_again(_B, 1), _again(_B, 3)]
# one stream, one tap, a window of one token, no rotation, one expert
_C = [_moe(_conv(2, 2, 48, 48, 0.2, 1), 32, 1.5, 1, 1),
      _moe(_parallel((3, 3, 16, 16, 0.6), 1, 0, None, (1, 130, 20), 2.0, (0.5, 0.25)), 28, 1.0, 4, 4, (2, 2)),
      _moe(_parallel((3, 1, 16, 48, 0.5), 64, 64, (16, 500.0), (6, 1, 1), 30.0, (1.5, -0.3)), 24, 3.0, 9, 2, (3, 1)),
      _moe(_biased(1, 1, 96, 16, 0.1), 36, 0.8, 3, 2)]
# many streams, a width that is no multiple of 8, a layer that uses a later layer's weights
_D = [_moe(_conv(4, 2, 12, 20, 0.5, 2), 12, 1.1, 6, 3, (2, 2)),
      _biased(6, 1, 6, 6, 0.8),
      _moe(_parallel((2, 2, 20, 4, 0.4), 17, 40, (4, 90.0), (2, 20, 33), 6.0, (1.0, 0.6)), 20, 0.7, 8, 2, (4, 1)),
      _moe(_conv(5, 5, 8, 8, 0.9, 5), 16, 5.0, 2, 2)]
_D = [_again(_D, 2)] + [dict(l) for l in _D]
_D[0]["weights_of"] = 3
_D += [dict(_D[2], weights_of=2)]

# every router gives a token all its experts: nothing to decide, so that rounding never leads to another computation
_F = [_moe(_parallel((4, 2, 32, 32, 0.2), 40, 20, (16, 2000.0), (4, 16, 16), 15.0, (1.0, 0.5)), 24, 1.2, 4, 4, (2, 2)),
      _moe(_conv(4, 1, 32, 48, 0.15, 4), 32, 3.0, 2, 2),
      _biased(4, 2, 64, 64, 0.1)]
_F += [_again(_F, 0)]

# name -> (config, seed, page size)
TINY_D: Dict[str, tuple] = {
    "A": (_cfg(83, 48, 2e-2, 3, _A, bigram=(37, 11, 5), softcap=9.0), 61, 8),
    "B": (_cfg(157, 64, 5e-2, 4, _B, bigram=(210, 13, 150), softcap=30.0), 62, 16),
    "C": (_cfg(120, 96, 1e-2, 1, _C), 63, 32),
    "D": (_cfg(61, 52, 3e-2, 5, _D, bigram=(1, 3, 0), softcap=4.0), 64, 16),
    "E": (_cfg(70, 40, 1e-5, 9, _A[:2], bigram=(64, 0, 1)), 65, 16),
    "F": (_cfg(131, 64, 2e-2, 4, _F, bigram=(99, 5, 17), softcap=12.0), 66, 16),
}


def sharpen(name: str, t: torch.Tensor):
    """Scores that spread over a few units: flat attention would hide a missing key, a sink or a wrong edge behind the
    tolerance, and sharper one would let the roundings of bfloat16 decide.  Filters of the size of one make a lost input of
    the convolution show; forget gates near one (a bias of a few units) let the memory reach far back; router logits of a few
    units keep its softmax off its ends; stream mixes near a permutation keep the streams apart without letting them
    grow."""
    leaf = name.rsplit(".", 1)[-1]
    if leaf in ("q", "k") and ".mix." in name:
        return t.float() * 0.9
    if name.endswith(".conv"):
        return t.float() * 0.7
    if name.endswith(".f.b"):
        return t.float() + 4.0
    if name.endswith(".router"):
        return t.float() * (1.2 / t.shape[1] ** 0.5)
    if name.endswith(".hc1.mix") or name.endswith(".hc2.mix"):
        n = t.shape[0]
        return 0.75 * torch.roll(torch.eye(n), 1, dims=1) + t.float() * 0.25 / n ** 0.5
    if name.endswith((".hc1.in", ".hc2.in")):
        return 0.4 * t.float() + 0.5
    if name.endswith((".hc1.out", ".hc2.out")):
        return 0.5 * t.float() + 0.7
    if name == "embed":
        return t.float() * 6.0
    return None


def make_folder(path: str, name: str, store_dtype=torch.float32, override=None) -> str:
    """config.json and model.safetensors with random weights large enough that every layer matters."""
    from xinfer_b200.weights import write_random_model
    cfg, seed, _ = TINY_D[name]

    def both(n, t):
        if override is not None:
            r = override(n, t)
            if r is not None:
                return r
        return sharpen(n, t)

    return write_random_model(path, cfg, seed, dtype=store_dtype, std=0.12, norm_std=0.2, override=both)


def prompts(name: str, lengths: Sequence[int], seed: int = 0) -> List[List[int]]:
    cfg = TINY_D[name][0]
    rng = np.random.default_rng(800 + seed)
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
