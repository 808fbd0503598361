"""Tiny Napuzen configurations for the tests (config.json dictionaries) and their random model folders.

They differ from each other in every size and switch: convolutions of one tap (no state), of two to five and of more
taps than the fused kernel takes; heads, key and value sizes that differ, that are one, that are no power of two;
decays of several time constants; latent ranks and query ranks that fit the tensor-core kernels and that do not;
rotations over all of the rotated part or half of it, with and without scaling; windows of one token, shorter and
longer than a page and no multiple of it; latent rows read by none, one and two other layers, with shorter and with
longer windows, also rows that carry a rotated part the reader has no use for; dense and routed feed-forwards and
layers without one; routers over one to twelve experts that give a token one, some or all of them, with and without the
shared expert; a width that is no multiple of 8; logit scales below and above one; vocabulary and page size."""
from typing import Dict, List, Sequence

import numpy as np
import torch


def _gla(heads, dim, vdim, tau):
    return dict(type="gla", mixer=dict(heads=heads, dim=dim, vdim=vdim, tau=tau))


def _latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, dims=None, scaling=None):
    rot = dict(dims=rot_dim if dims is None else dims, base=base)
    if scaling is not None:
        rot["scaling"] = scaling
    return dict(type="latent_attention", mixer=dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank,
                                                    kv_rank=kv_rank, scale=scale, rot=rot))


def _latent2(heads, dim, vdim, kv_rank, scale, window, kv_from=None):
    m = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, scale=scale, mask=dict(size=window))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention_2", mixer=m)


def _dense(layer, ff, limit):
    return dict(layer, mlp=dict(kind="dense", ff=ff, limit=limit))


def _none(layer):
    return dict(layer, mlp=None)


def _moe(layer, ff, experts, top, scale, shared=None):
    mlp = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if shared is not None:
        mlp["shared"] = dict(ff=shared)
    return dict(layer, mlp=mlp)


def _cfg(vocab, width, eps, taps, logit_scale, layers):
    return dict(architecture="Napuzen", vocab=vocab, width=width, norm=dict(eps=eps), canon=dict(taps=taps),
                logit_scale=logit_scale, layers=layers)


_YARN = dict(factor=3.0, original=64, fast=4.0, slow=0.5)

# name -> (config, seed, page size)
TINY_N: Dict[str, tuple] = {
    # sizes that fit no fast path, a reader with a longer window than the owner's
    "N1": (_cfg(83, 48, 1e-5, 4, 0.7, [
        _moe(_gla(3, 10, 14, 4.0), 24, 5, 2, 1.5, shared=20),
        _dense(_latent2(3, 12, 10, 20, 0.6, 11), 40, 1.2),
        _none(_gla(1, 7, 5, 1.0)),
        _moe(_latent(5, 6, 4, 9, 18, 14, 0.5, 50.0, scaling=_YARN), 16, 7, 7, 0.8, shared=12),
        _dense(_latent2(2, 9, 16, 20, 0.25, 37, kv_from=1), 24, 0.7),
    ]), 51, 8),
    # sizes of the tensor-core kernels, a latent read twice, two taps, all experts of a router of one
    "N2": (_cfg(157, 64, 3e-6, 2, 1.8, [
        _dense(_latent(4, 16, 16, 32, 48, 48, 0.4, 30000.0, scaling=dict(factor=4.0, original=96, fast=16.0, slow=1.0)), 96, 2.5),
        _moe(_gla(4, 32, 16, 16.0), 32, 12, 4, 2.5, shared=48),
        _moe(_latent2(8, 24, 16, 64, 0.11, 50), 40, 1, 1, 1.0),
        _moe(_latent2(4, 16, 24, 64, 0.13, 23, kv_from=2), 48, 6, 1, 3.0, shared=16),
        _none(_latent2(2, 32, 32, 64, 0.07, 130, kv_from=2)),
    ]), 52, 16),
    # more taps than the fused kernel takes, a reader of rows with a rotated part, rotation over half of it
    "N3": (_cfg(120, 96, 1e-6, 11, 0.4, [
        _moe(_latent(2, 24, 8, 20, 32, 40, 0.8, 1000.0, dims=4), 32, 4, 2, 1.2, shared=64),
        _dense(_gla(2, 48, 40, 8.0), 72, 3.0),
        _moe(_latent2(6, 20, 12, 40, 0.09, 64, kv_from=0), 24, 9, 3, 2.0),
        _none(_latent2(1, 40, 8, 56, 0.05, 1)),
    ]), 53, 32),
    # one tap, a width that is no multiple of 8, attention last, no routers but one
    "N4": (_cfg(61, 52, 2e-6, 1, 1.0, [
        _dense(_gla(5, 4, 20, 2.0), 36, 1.5),
        _none(_latent(3, 10, 6, 6, 12, 24, 0.6, 300.0)),
        _moe(_latent2(4, 8, 12, 28, 0.35, 17), 12, 3, 2, 0.5, shared=8),
        _dense(_gla(2, 20, 6, 32.0), 28, 0.9),
    ]), 54, 16),
}


def sharpen(name: str, t: torch.Tensor):
    """Random N(0, std) weights give nearly flat attention, which would hide a missing key or a wrong edge behind the
    tolerance.  Larger weights on the cached latents' norms spread the scores over a few units; filters of the size of
    one make a lost input of the convolution show; router logits of a few units keep its softmax off its ends; a smaller
    embedding keeps the tied head from repeating the last token."""
    if name.endswith(".dkv.norm"):
        return t.float() * 2.5
    if name.endswith(".canon1"):
        return t.float() * 2.0
    if name.endswith(".router") or name.endswith(".shared.sg"):
        return t.float() * (1.0 / t.shape[1] ** 0.5)
    if name == "embed":
        return t.float() * 0.6
    return None


def make_folder(path: str, name: str, store_dtype=torch.float32, override=None) -> str:
    """config.json and model.safetensors with random weights large enough that every layer matters."""
    from xinfer_b200.weights import write_random_model
    cfg, seed, _ = TINY_N[name]

    def both(n, t):
        if override is not None:
            r = override(n, t)
            if r is not None:
                return r
        return sharpen(n, t)

    return write_random_model(path, cfg, seed, dtype=store_dtype, std=0.12, norm_std=0.2, override=both)


def prompts(name: str, lengths: Sequence[int], seed: int = 0) -> List[List[int]]:
    cfg = TINY_N[name][0]
    rng = np.random.default_rng(700 + seed)
    return [rng.integers(0, cfg["vocab"], size=n).tolist() for n in lengths]
