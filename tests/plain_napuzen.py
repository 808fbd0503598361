"""A plain, slow implementation of the Napuzen decoder: float64, whole sequences at once, one function per
mechanism, written from the design's equations.  It shares no code with the engine (it even reads model folders
itself) and serves as the oracle of the tests.

    x_0    = E[token]
    layer:   x <- x + N1(mixer(c(x)));  x <- x + N2(ff(x))         norms behind the sublayers, none in front
             c(x)_t = x_t + sum_j taps[:, j] * x_(t - K + 1 + j)     a causal convolution beside the identity
    logits = E . Nf(x) * logit_scale

``round_to`` emulates an engine that stores activations in a shorter type: the inputs of the sublayers, the results
of matrix products that an engine keeps in that type, the cached rows, the queries and the heads' outputs are rounded
to it and widened again; what belongs to a recurrence, a norm, a router or the stream stays wide.
"""
import json
import math
import os
import struct

import numpy as np
import torch

F64 = torch.float64
SWISH_ALPHA = 1.702       # fixed by the design


# ---- model folders --------------------------------------------------------------------------------------------------
def load_folder(folder):
    """(config dict, {name: float64 tensor}) of a folder with config.json and model.safetensors."""
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    with open(os.path.join(folder, "model.safetensors"), "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    w = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        raw = torch.from_numpy(np.frombuffer(data[a:b], dtype=np.uint8).copy())
        kind = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32}[e["dtype"]]
        t = raw.view(kind).reshape(e["shape"])
        w[name] = t.to(torch.int64) if kind == torch.int32 else t.to(F64)
    return cfg, w


def _r(t, round_to):
    return t if round_to is None else t.to(round_to).to(F64)


# ---- norm and convolution -----------------------------------------------------------------------------------------------
def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * weight


def causal_conv(x, taps):
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, j] x_(t - K + 1 + j), inputs before the sequence are zero."""
    T, C = x.shape
    K = taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for j in range(K):
        y += taps[:, j] * padded[j:j + T]
    return y


# ---- gated linear attention ---------------------------------------------------------------------------------------------
def key_decay(z, tau):
    """sigmoid(z)^(1 / tau)."""
    return torch.sigmoid(z) ** (1.0 / tau)


def linear_recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, H, d], v [T, H, dv] -> (o [T, H, dv], S [H, d, dv]).  S <- diag(alpha_t) S + k_t v_t^T and
    o_t = S^T q_t, one token after the other; the read sees the token's own write."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64) if state is None else state.clone()
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return o, S


def gla_mixer(h, w, p, m, eps, round_to=None):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    q, k, v = _r(q, round_to), _r(k, round_to), _r(v, round_to)
    z = _r(h @ w[p + "a1"].T, round_to) @ w[p + "a2"].T + w[p + "a2.b"]
    o, _ = linear_recurrence(q, k, v, key_decay(z.view(T, H, d), m["tau"]))
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, H * dv)
    g = _r(h @ w[p + "g"].T, round_to)
    return _r(o * g * torch.sigmoid(g), round_to) @ w[p + "o"].T


# ---- rotation -----------------------------------------------------------------------------------------------------------
def yarn_frequencies(dims, base, scaling):
    """(frequency of every pair, factor on cos and sin)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return torch.tensor(f, dtype=F64), 1.0

    def at(turns):
        return dims * math.log(scaling["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(at(scaling["fast"])), 0)
    hi = min(math.ceil(at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_neighbours(x, positions, rot):
    """x [T, heads, d]: channels (2i, 2i+1) of the first rot.dims turn by position * f_i; the rest pass."""
    f, mag = yarn_frequencies(rot["dims"], rot["base"], rot.get("scaling"))
    a = positions.to(F64)[:, None] * f[None, :]
    c, s = mag * torch.cos(a)[:, None, :], mag * torch.sin(a)[:, None, :]
    n = rot["dims"]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * c - v * s
    out[..., 1:n:2] = v * c + u * s
    return out


# ---- attention over a cached latent -----------------------------------------------------------------------------------
def causal_mask(T, window=None):
    """[T, T] True where query i sees key j: 0 <= i - j (< window)."""
    dist = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (dist >= 0) if window is None else (dist >= 0) & (dist < window)


def softmax_heads(q, k, v, mask, scale):
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv]; ordinary softmax over the keys the mask shows."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=F64)
    for h in range(q.shape[1]):
        s = ((q[:, h] @ k[:, h].T) * scale).masked_fill(~mask, -math.inf)
        out[:, h] = torch.softmax(s, dim=-1) @ v[:, h]
    return out


def latent_rows(h, w, p, rank, eps, positions, rot=None, round_to=None):
    """What a token caches: (c [T, rank], rotated key part [T, rot_dim] or None)."""
    kv = _r(h @ w[p + "dkv"].T, round_to)
    c = _r(rms_norm(kv[:, :rank], w[p + "dkv.norm"], eps), round_to)
    if rot is None:
        return c, None
    return c, _r(rotate_neighbours(kv[:, None, rank:], positions, rot)[:, 0], round_to)


def latent_mixer(h, w, p, m, eps, positions, round_to=None):
    """The mixer 'latent_attention': queries through a latent of their own, a rotated part, every earlier key."""
    T = h.shape[0]
    H, d, rd, dv, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    cq = _r(rms_norm(_r(h @ w[p + "dq"].T, round_to), w[p + "dq.norm"], eps), round_to)
    q = _r(cq @ w[p + "uq"].T, round_to).view(T, H, d + rd)
    q = torch.cat([q[..., :d], _r(rotate_neighbours(q[..., d:], positions, m["rot"]), round_to)], dim=-1)
    c, kr = latent_rows(h, w, p, r, eps, positions, m["rot"], round_to)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, d), kr[:, None, :].expand(T, H, rd)], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = softmax_heads(q, k, v, causal_mask(T), m["scale"])
    return _r(o.reshape(T, H * dv), round_to) @ w[p + "o"].T, c


def gated_latent_mixer(h, w, p, m, eps, positions, shared_rows=None, round_to=None):
    """The mixer 'latent_attention_2': no positions, a window, a gate of one number per head; ``shared_rows``: the
    latent of the layer whose cache this one reads."""
    T = h.shape[0]
    H, d, dv, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
    q = _r(h @ w[p + "q"].T, round_to).view(T, H, d)
    c = shared_rows if shared_rows is not None else latent_rows(h, w, p, r, eps, positions, None, round_to)[0]
    k = (c @ w[p + "uk"].T).view(T, H, d)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = softmax_heads(q, k, v, causal_mask(T, m["mask"]["size"]), m["scale"])
    gate = torch.sigmoid(_r(h @ w[p + "g"].T, round_to))
    return _r((o * gate[:, :, None]).reshape(T, H * dv), round_to) @ w[p + "o"].T, c


# ---- feed-forwards ------------------------------------------------------------------------------------------------------
def clamped_feed_forward(h, w, p, limit, round_to=None):
    g = _r(h @ w[p + "gate"].T, round_to).clamp(max=limit)
    u = _r(h @ w[p + "up"].T, round_to).clamp(-limit, limit)
    return _r(g * torch.sigmoid(SWISH_ALPHA * g) * (u + 1.0), round_to) @ w[p + "down"].T


def silu_expert(h, w, p, round_to=None):
    g = _r(h @ w[p + "gate"].T, round_to)
    u = _r(h @ w[p + "up"].T, round_to)
    return _r(g * torch.sigmoid(g) * u, round_to) @ w[p + "down"].T


def route(h, w_router, top, scale):
    """(chosen experts [T, top] by falling score, their weights [T, top]): scores softmax(W_r h) over all experts;
    weights the chosen scores over their sum, times scale."""
    s = torch.softmax(h @ w_router.T, dim=-1)
    wt, idx = s.topk(top, dim=-1)
    return idx, wt / (wt.sum(-1, keepdim=True) + 1e-20) * scale


def follow_close_calls(h, w_router, scale, idx, wt, given, slack):
    """An engine that rounds activations may decide a close call the other way.  ``given`` [T, top] are the experts
    an engine chose: where a token's set differs from the plain one, every expert it took instead must have a logit
    within ``slack`` of one it left out - else the engine's router is wrong and this raises.  Returns the engine's
    sets with their plain weights."""
    z = h @ w_router.T
    s = torch.softmax(z, dim=-1)
    out_i, out_w = idx.clone(), wt.clone()
    for t in range(z.shape[0]):
        mine, theirs = set(idx[t].tolist()), set(int(e) for e in given[t].tolist())
        if mine == theirs:
            continue
        assert len(theirs) == len(mine), f"token {t}: the engine chose {sorted(theirs)}"
        for e in theirs - mine:
            near = min(abs(float(z[t, e] - z[t, o])) for o in mine - theirs)
            assert near <= slack, f"token {t}: expert {e} instead of one of {sorted(mine - theirs)} is no close call ({near:.3g})"
        order = sorted(theirs, key=lambda e: -float(z[t, e]))
        out_i[t] = torch.tensor(order)
        out_w[t] = s[t, order] / (s[t, order].sum() + 1e-20) * scale
    return out_i, out_w


def routed_experts(h, w, p, mlp, round_to=None, given=None, slack=0.0):
    r = mlp["router"]
    idx, wt = route(h, w[p + "router"], r["top"], r["scale"])
    if given is not None:
        idx, wt = follow_close_calls(h, w[p + "router"], r["scale"], idx, wt, given, slack)
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=F64)
    for e in range(r["experts"]):
        rows, j = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += wt[rows, j][:, None] * silu_expert(h[rows], w, f"{p}e{e}.", round_to)
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(h @ w[p + "shared.sg"].T) * silu_expert(h, w, p + "shared.", round_to)
    return out


def feed_forward(h, w, p, mlp, round_to=None, given=None, slack=0.0):
    if mlp["kind"] == "dense":
        return clamped_feed_forward(h, w, p, mlp["limit"], round_to)
    return routed_experts(h, w, p, mlp, round_to, given, slack)


# ---- the whole model ------------------------------------------------------------------------------------------------------
def forward(cfg, w, tokens, round_to=None, streams=None, routes=None, slack=0.0):
    """float64 logits [T, vocab] of one sequence; ``streams`` (a list) receives the residual stream after every
    layer.  ``routes``: per layer (None where it has no router) the experts an engine chose, [T, top]: they are
    followed where they differ from the plain choice by close calls only (``follow_close_calls``)."""
    tokens = torch.as_tensor(tokens, dtype=torch.int64)
    positions = torch.arange(tokens.shape[0])
    eps = cfg["norm"]["eps"]
    x = w["embed"][tokens]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = _r(x + causal_conv(x, w[p + "canon1"]), round_to)
        if layer["type"] == "gla":
            a = gla_mixer(h, w, p + "mix.", m, eps, round_to)
        elif layer["type"] == "latent_attention":
            a, latents[i] = latent_mixer(h, w, p + "mix.", m, eps, positions, round_to)
        elif layer["type"] == "latent_attention_2":
            rows = latents[m["kv_from"]] if m.get("kv_from") is not None else None
            a, latents[i] = gated_latent_mixer(h, w, p + "mix.", m, eps, positions, rows, round_to)
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(a, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            given = routes[i] if routes is not None else None
            f = feed_forward(_r(x, round_to), w, p + "mlp.", layer["mlp"], round_to, given, slack)
            x = x + rms_norm(f, w[p + "norm2"], eps)
        if streams is not None:
            streams.append(x.clone())
    y = _r(rms_norm(x, w["final.norm"], eps), round_to)
    return y @ w["embed"].T * cfg["logit_scale"]


def greedy(cfg, w, prompt, n):
    """Greedy continuation by n tokens, the whole sequence computed again for every token."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
