"""A plain, slow implementation of the Dalalix decoder: float64, whole sequences at once, one function per mechanism,
written from the design's equations.  It shares no code with the engine (it even reads model folders itself) and serves
as the oracle of the tests.

    X_0[s]  = E[token] + P[pair row]                        the same in every one of the n streams
    half a layer:   u = sum_s r_s X[s];   y = sublayer(N(u));   X[t] <- sum_s M[s, t] X[s] + w_t y
    logits  = cap tanh( W_head Nf(sum_s X[s]) / cap )

``round_to`` emulates an engine that stores activations in a shorter type: the inputs of the sublayers, the projections
of attention, its queries, keys, values and outputs and the experts' activations are rounded to it and widened again;
what belongs to a recurrence, a norm, a router or the streams stays wide.
"""
import json
import math
import os
import struct

import numpy as np
import torch

F64 = torch.float64
SWISH_ALPHA = 1.702       # fixed by the design
MEMORY_EPS = 1e-6         # beside the matrix memory's divisor
WEIGHT_SUM_EPS = 1e-20    # beside the sum of a token's chosen scores


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


# ---- small pieces ---------------------------------------------------------------------------------------------------
def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps under the root."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def causal_conv(x, taps):
    """x [T, C], taps [C, K]: y_t = sum_j taps[:, j] x_(t - K + 1 + j), inputs before the sequence are zero."""
    T, C = x.shape
    K = taps.shape[1]
    padded = torch.cat([torch.zeros(K - 1, C, dtype=x.dtype), x])
    y = torch.zeros_like(x)
    for j in range(K):
        y += taps[:, j] * padded[j:j + T]
    return y


# ---- embedding ------------------------------------------------------------------------------------------------------
def pair_rows(tokens, rule):
    """A row of the pair table per token: a hash of (token before, token), the last row for the first token."""
    out = [rule["buckets"]]
    for a, b in zip(tokens[:-1], tokens[1:]):
        out.append((a * rule["mul_prev"] + b * rule["mul_cur"]) % rule["buckets"])
    return out


def embed(cfg, w, tokens):
    x = w["embed"][torch.tensor(tokens)]
    rule = (cfg.get("embedding") or {}).get("bigram")
    if rule is not None:
        x = x + w["bigram"][torch.tensor(pair_rows(list(tokens), rule))]
    return x


# ---- several residual streams ---------------------------------------------------------------------------------------
def read_streams(X, r):
    """X [n, T, W], r [n] -> [T, W]."""
    return torch.einsum("s,stw->tw", r, X)


def write_streams(X, M, w, y):
    """All n streams at once from the old ones: X'[t] = sum_s M[s, t] X[s] + w[t] y."""
    return torch.einsum("st,sab->tab", M, X) + w[:, None, None] * y


# ---- softmax attention ----------------------------------------------------------------------------------------------
def rotate_halves(x, positions, dims, base):
    """x [T, heads, d]: channel i of the first dims/2 pairs with channel i + dims/2 and turns by position * f_i."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=F64)
    a = positions.to(F64)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T, window=None, keep_first=0):
    """[T, T] True where query i sees key j: not later, and less than ``window`` back or among the first
    ``keep_first``."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    m = j <= i
    if window is not None:
        m = m & ((i - j < window) | (j < keep_first))
    return m


def softmax_heads(q, k, v, mask, scale, sink=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; query head h reads head h // (H / G).  ``sink`` [H]: one
    more entry of that score in every softmax of the head, without a value."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for h in range(H):
        s = ((q[:, h] @ k[:, h // rep].T) * scale).masked_fill(~mask, -math.inf)
        if sink is not None:
            s = torch.cat([s, torch.full((T, 1), float(sink[h]), dtype=F64)], dim=1)
        out[:, h] = torch.softmax(s, dim=-1)[:, :T] @ v[:, h // rep]
    return out


def conv_attention(h, w, p, m, eps, round_to=None):
    """The mixer 'attention': convolved projections, values of unit size, every earlier key, a sigmoid gate per
    channel."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (causal_conv(_r(h @ w[p + n].T, round_to), w[p + n + ".conv"]) for n in ("q", "k", "v"))
    q, k = _r(q, round_to).view(T, H, d), _r(k, round_to).view(T, G, d)
    v = _r(unit_rms(v.view(T, G, dv), eps), round_to)
    o = _r(softmax_heads(q, k, v, visible(T), m["scale"]).reshape(T, H * dv), round_to)
    g = torch.sigmoid(_r(h @ w[p + "g"].T, round_to))
    return _r(o * g, round_to) @ w[p + "o"].T


def biased_attention(h, w, p, m, positions, window=None, keep_first=0, sink=None, rot=None, round_to=None):
    """Attention with biases on q, k and v: the mixer 'attention_2', and with a rotation, a window that keeps the first
    tokens and a sink the left side of the mixer 'parallel'.  Without the output projection: [T, heads * vdim]."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (_r(h @ w[p + n].T, round_to) + w[p + n + ".b"] for n in ("q", "k", "v"))
    q, k, v = q.view(T, H, d), k.view(T, G, d), v.view(T, G, dv)
    if rot is not None and rot["dims"]:
        q, k = (rotate_halves(x, positions, rot["dims"], rot["base"]) for x in (q, k))
    q, k, v = _r(q, round_to), _r(k, round_to), _r(v, round_to)
    return softmax_heads(q, k, v, visible(T, window, keep_first), m["scale"], sink).reshape(T, H * dv)


# ---- matrix memory --------------------------------------------------------------------------------------------------
def memory_gates(zi, zf, cap):
    """(log input gate, log forget gate) from the biased pre-activations."""
    return cap * torch.tanh(zi / cap), torch.nn.functional.logsigmoid(cap * torch.tanh(zf / cap))


def memory_recurrence(q, k, v, i, f, state=None):
    """q, k [T, H, d], v [T, H, dv], i, f [T, H] (logarithms) -> (o [T, H, dv], (S, n, m)), one token after the other:

        m' = max(f + m, i);  S' = e^(f + m - m') S + e^(i - m') k v^T;  n' = e^(f + m - m') n + e^(i - m') k
        o  = S'^T q / (max(|n' . q|, e^(-m')) + 1e-6)

    S, n and m start at zero."""
    T, H, d = q.shape
    if state is None:
        S, n, m = torch.zeros(H, d, v.shape[2], dtype=F64), torch.zeros(H, d, dtype=F64), torch.zeros(H, dtype=F64)
    else:
        S, n, m = (t.clone() for t in state)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        m2 = torch.maximum(f[t] + m, i[t])
        a, b = torch.exp(f[t] + m - m2), torch.exp(i[t] - m2)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = a[:, None] * n + b[:, None] * k[t]
        m = m2
        div = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + MEMORY_EPS
        o[t] = torch.einsum("hdv,hd->hv", S, q[t]) / div[:, None]
    return o, (S, n, m)


def memory_mixer(h, w, p, m, eps, round_to=None):
    """The right side of the mixer 'parallel' without its output projection: [T, heads * vdim]."""
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w[p + "k"].T).view(T, H, d)
    v = (h @ w[p + "v"].T).view(T, H, dv)
    q, k, v = _r(q, round_to), _r(k, round_to), _r(v, round_to)
    i, f = memory_gates(h @ w[p + "i"].T + w[p + "i.b"], h @ w[p + "f"].T + w[p + "f.b"], m["gate_cap"])
    o, _ = memory_recurrence(q, k, v, i, f)
    g = torch.sigmoid(_r(h @ w[p + "g"].T, round_to))
    return unit_rms(o, eps).reshape(T, H * dv) * w[p + "norm"] * g


def parallel_mixer(h, w, p, m, eps, positions, round_to=None):
    a, b = m["left"], m["right"]
    lo = biased_attention(h, w, p + "left.", a, positions, a["mask"]["size"], a["mask"]["keep_first"], w[p + "left.sink"],
                          a.get("rot"), round_to)
    ro = memory_mixer(h, w, p + "right.", b, eps, round_to)
    return (_r(lo * m["left_scale"], round_to) @ w[p + "left.o"].T + _r(ro * m["right_scale"], round_to) @ w[p + "right.o"].T)


# ---- experts --------------------------------------------------------------------------------------------------------
def expert(h, w, p, limit, round_to=None):
    g = _r(h @ w[p + "gate"].T, round_to).clamp(max=limit)
    u = _r(h @ w[p + "up"].T, round_to).clamp(-limit, limit)
    return _r(g * torch.sigmoid(SWISH_ALPHA * g) * (u + 1.0), round_to) @ w[p + "down"].T


def allowed_experts(s, groups, keep):
    """[T, E] True for the experts of the ``keep`` groups of neighbours whose best score is largest."""
    T, E = s.shape
    best = s.view(T, groups, E // groups).max(dim=-1).values
    kept = torch.zeros(T, groups, dtype=torch.bool)
    kept.scatter_(1, best.topk(keep, dim=-1).indices, True)
    return kept[:, :, None].expand(T, groups, E // groups).reshape(T, E)


def group_rule(router):
    g = router.get("groups") or {"count": 1, "keep": 1}
    return g["count"], g["keep"]


def route(h, w_router, router):
    """(chosen experts [T, top] by falling score, their weights [T, top])."""
    s = torch.softmax(h @ w_router.T, dim=-1)
    c = s.masked_fill(~allowed_experts(s, *group_rule(router)), -math.inf)
    idx = c.topk(router["top"], dim=-1).indices
    wt = s.gather(1, idx)
    return idx, wt / (wt.sum(-1, keepdim=True) + WEIGHT_SUM_EPS)


def follow_close_calls(h, w_router, router, idx, wt, given, slack):
    """An engine that rounds activations may decide a close call the other way.  ``given`` [T, top] are the experts an
    engine chose: where a token's set differs from the plain one, the engine's set must be what the rule gives for
    logits that are off by at most ``slack`` - else the engine's router is wrong and this raises.  Returns the engine's
    sets with their plain weights."""
    z = h @ w_router.T
    s = torch.softmax(z, dim=-1)
    groups, keep = group_rule(router)
    per = z.shape[1] // groups
    out_i, out_w = idx.clone(), wt.clone()
    for t in range(z.shape[0]):
        mine, theirs = set(idx[t].tolist()), set(int(e) for e in given[t].tolist())
        if mine == theirs:
            continue
        assert len(theirs) == len(mine), f"token {t}: the engine chose {sorted(theirs)}"
        # push the engine's experts up and the others down by the slack: the rule must then give the engine's set.  (A
        # group that was close is decided by its best expert, which may itself be no chosen one: a group that holds an
        # expert of the engine's is pushed up as a whole.)
        up = torch.full_like(z[t], -slack)
        for e in theirs:
            up[e // per * per:(e // per + 1) * per] = 0.0
        for e in theirs:
            up[e] = slack
        zz = (z[t] + up)[None]
        best = zz.view(1, groups, per).max(dim=-1).values
        kept = set(best.topk(keep, dim=-1).indices[0].tolist())
        allowed = [e for e in range(z.shape[1]) if e // per in kept]
        got = set(sorted(allowed, key=lambda e: -float(zz[0, e]))[:len(theirs)])
        assert got == theirs, f"token {t}: {sorted(theirs)} instead of {sorted(mine)} is no close call"
        order = sorted(theirs, key=lambda e: -float(z[t, e]))
        out_i[t] = torch.tensor(order)
        out_w[t] = s[t, order] / (s[t, order].sum() + WEIGHT_SUM_EPS)
    return out_i, out_w


def routed_experts(h, w, p, mlp, round_to=None, given=None, slack=0.0):
    r = mlp["router"]
    idx, wt = route(h, w[p + "router"], r)
    if given is not None:
        idx, wt = follow_close_calls(h, w[p + "router"], r, idx, wt, given, slack)
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=F64)
    for e in range(r["experts"]):
        rows, j = (idx == e).nonzero(as_tuple=True)
        if len(rows):
            out[rows] += wt[rows, j][:, None] * expert(h[rows], w, f"{p}e{e}.", mlp["expert"]["limit"], round_to)
    return out


# ---- the whole model ------------------------------------------------------------------------------------------------
def mixer(h, w, p, layer, eps, positions, round_to=None):
    m = layer["mixer"]
    if layer["type"] == "attention":
        return conv_attention(h, w, p, m, eps, round_to)
    if layer["type"] == "attention_2":
        return _r(biased_attention(h, w, p, m, positions, round_to=round_to), round_to) @ w[p + "o"].T
    if layer["type"] == "parallel":
        return parallel_mixer(h, w, p, m, eps, positions, round_to)
    raise ValueError(layer["type"])


def forward(cfg, w, tokens, round_to=None, streams=None, routes=None, slack=0.0):
    """float64 logits [T, vocab] of one sequence; ``streams`` (a list) receives the sum of the residual streams after
    every layer.  ``routes``: per layer (None where it has no router) the experts an engine chose, [T, top]: they are
    followed where they differ from the plain choice by close calls only (``follow_close_calls``)."""
    tokens = [int(t) for t in tokens]
    positions = torch.arange(len(tokens))
    eps = cfg["norm"]["eps"]
    x = embed(cfg, w, tokens)
    X = x[None].repeat(cfg["streams"], 1, 1)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer['weights_of'] if layer.get('weights_of') is not None else i}."
        h = _r(rms_norm(read_streams(X, w[p + "hc1.in"]), w[p + "norm1"], eps), round_to)
        y = mixer(h, w, p + "mix.", layer, eps, positions, round_to)
        X = write_streams(X, w[p + "hc1.mix"], w[p + "hc1.out"], y)
        if layer.get("mlp") is not None:
            h = _r(rms_norm(read_streams(X, w[p + "hc2.in"]), w[p + "norm2"], eps), round_to)
            y = routed_experts(h, w, p + "mlp.", layer["mlp"], round_to, routes[i] if routes is not None else None, slack)
            X = write_streams(X, w[p + "hc2.mix"], w[p + "hc2.out"], y)
        if streams is not None:
            streams.append(X.sum(dim=0))
    y = _r(rms_norm(X.sum(dim=0), w["final.norm"], eps), round_to)
    logits = y @ w["head"].T
    cap = cfg.get("logit_softcap")
    return logits if cap is None else cap * torch.tanh(logits / cap)


def greedy(cfg, w, prompt, n):
    """Greedy continuation by n tokens, the whole sequence computed again for every token."""
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]
