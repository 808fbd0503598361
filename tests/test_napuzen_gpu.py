"""The Napuzen decoder on the GPU against the plain implementation (plain_napuzen.py): every mechanism alone through
its kernel, then whole models through the step function, the replay program and the generation entry point - whole
prompts, token-by-token decoding, portions down to two tokens, unequal batches, pages and slots that are used again,
keys far back and at the edges of windows and pages, the first tokens of a sequence."""
import numpy as np
import pytest
import torch

import plain_napuzen as plain
from napuzen_models import TINY_N, make_folder, prompts
from helpers import build_all_modes, replay_with_routes, row_error, run_trace

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64


def _k():
    from xinfer_b200 import kernels
    return kernels


def _err():
    return torch.zeros(1, dtype=torch.int32, device=DEV)


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device=DEV)


def _rand(*shape, seed=0, scale=1.0):
    return torch.randn(tuple(shape), generator=torch.Generator().manual_seed(seed), dtype=F64) * scale


def _tol(dtype):
    return 2e-5 if dtype == torch.float32 else 3e-2


def _batch(counts, slots):
    """(req_of_token, q_start, slots) of a step whose entries bring ``counts`` tokens (an entry of None: one padding
    token)."""
    req, starts, real = [], [0], []
    for b, n in enumerate(counts):
        req += [-1] if n is None else [b] * n
        starts.append(len(req))
    return _i32(req), _i32(starts), _i32(slots)


# ---------------------------------------------------------------------------------------------
# the convolution beside the identity, with the stream's sum in the same pass
# ---------------------------------------------------------------------------------------------
def _stream_conv_steps(C, K, lens, cuts, dtype, branch, seed, norm=True, scale=1.0):
    """Runs requests of ``lens`` tokens through the kernel in steps: ``cuts`` lists the steps, each a list of
    (request, tokens).  Returns per request (out, sum) as the kernel gave them and as the plain functions do."""
    k = _k()
    eps = 1e-5
    xs = [_rand(n, C, seed=seed + 10 * i).float() for i, n in enumerate(lens)]
    bs = [_rand(n, C, seed=seed + 10 * i + 1, scale=3.0).float() for i, n in enumerate(lens)]
    w = (1 + _rand(C, seed=seed + 2, scale=0.3)).float()
    taps = _rand(C, K, seed=seed + 3, scale=0.5).float()
    slots = [(3 * i + 1) % (len(lens) + 2) for i in range(len(lens))]
    state = torch.zeros(len(lens) + 2, max(K - 1, 1), C, device=DEV)
    for s in slots:
        state[s].zero_()
    at = [0] * len(lens)
    outs, sums = [[] for _ in lens], [[] for _ in lens]
    for step in cuts:
        rows = [(r, at[r], at[r] + n) for r, n in step]
        req, q_start, sl = _batch([n for _, n in step], [slots[r] for r, _ in step])
        x = torch.cat([xs[r][a:b] for r, a, b in rows]).to(DEV)
        kw = {}
        if branch:
            total = torch.full_like(x, float("nan"))
            kw = dict(branch=torch.cat([bs[r][a:b] for r, a, b in rows]).to(DEV), sum_out=total, branch_scale=scale)
            if norm:
                kw.update(branch_weight=w.to(DEV), branch_eps=eps)
        out = torch.full(x.shape, float("nan"), dtype=dtype, device=DEV)
        k.stream_conv(out, x, taps.to(DEV), state if K > 1 else None, req, q_start, sl, len(step),
                      single=all(n == 1 for _, n in step), **kw)
        o = out.double().cpu()
        t = kw["sum_out"].double().cpu() if branch else x.double().cpu()
        i = 0
        for r, a, b in rows:
            outs[r].append(o[i:i + b - a])
            sums[r].append(t[i:i + b - a])
            i += b - a
            at[r] = b
    assert at == list(lens)
    want = []
    for x, b in zip(xs, bs):
        s = x.double()
        if branch:
            s = s + scale * (plain.rms_norm(b.double(), w.double(), eps) if norm else b.double())
        want.append((s + plain.causal_conv(s, taps.double()), s))
    return [(torch.cat(o), torch.cat(t)) for o, t in zip(outs, sums)], want


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("branch", [False, True])
@pytest.mark.parametrize("C,K", [(48, 4), (52, 2), (37, 3), (64, 1), (1200, 5), (33, 8)])
def test_convolution_however_the_tokens_are_cut(C, K, branch, dtype):
    lens = [23, 9, 40]
    whole = [[(0, 23), (1, 9), (2, 40)]]
    cut = [[(0, 2), (2, 1)], [(1, 1), (0, 3), (2, 5)], [(2, 1), (1, 1), (0, 1)], [(0, 17), (1, 7)], [(2, 2)], [(2, 31)]]
    singles = [[(2, 8), (0, 14)]] + [[(2, 1), (1, 1), (0, 1)]] * 9 + [[(2, 1)]] * 23
    for cuts in (whole, cut, singles):
        got, want = _stream_conv_steps(C, K, lens, cuts, dtype, branch, seed=C + K)
        for (o, s), (ro, rs) in zip(got, want):
            assert (s - rs).abs().max() <= 1e-5 * (1 + rs.abs().max())
            assert (o - ro).abs().max() <= (1e-5 if dtype == torch.float32 else 6e-3) * (1 + ro.abs().max())


def test_convolution_of_more_taps_than_the_fused_kernel_takes():
    k = _k()
    got, want = _stream_conv_steps(40, k.STREAM_CONV_FUSED_TAPS + 3, [30, 5], [[(0, 4), (1, 5)], [(0, 1)], [(0, 25)]],
                                   torch.float32, False, seed=5)
    for (o, _), (ro, _) in zip(got, want):
        assert (o - ro).abs().max() <= 1e-5 * (1 + ro.abs().max())
    with pytest.raises(k.KernelError):
        _stream_conv_steps(40, k.STREAM_CONV_FUSED_TAPS + 1, [4], [[(0, 4)]], torch.float32, True, seed=5)


@pytest.mark.parametrize("norm,scale", [(True, 0.5), (False, 1.0), (False, -0.7)])
def test_convolution_over_steps_of_thousands_of_tokens(norm, scale):
    """Blocks then take runs of several tokens that cross from one request into the next."""
    lens = [1501, 3, 1, 1030, 7]
    got, want = _stream_conv_steps(72, 4, lens, [[(i, n) for i, n in enumerate(lens)]], torch.float32, True, seed=9, norm=norm,
                                   scale=scale)
    for (o, s), (ro, rs) in zip(got, want):
        assert (s - rs).abs().max() <= 1e-5 * (1 + rs.abs().max()) and (o - ro).abs().max() <= 1e-5 * (1 + ro.abs().max())


def test_convolution_padding_tokens_leave_states_alone_and_stay_finite():
    k = _k()
    C, K = 40, 3
    state = _rand(3, K - 1, C, seed=1).float().to(DEV)
    before = state.clone()
    x = _rand(3, C, seed=2).float().to(DEV)
    out = torch.full_like(x, float("nan"))
    # one real request in slot 1, two padding tokens with slot -1
    k.stream_conv(out, x, _rand(C, K, seed=3).float().to(DEV), state, _i32([0, -1, -1]), _i32([0, 1, 1, 1]), _i32([1, -1, -1]), 3,
                  single=True)
    assert torch.equal(state[0], before[0]) and torch.equal(state[2], before[2]) and torch.isfinite(out).all()
    assert torch.equal(state[1, 1], x[0]) and torch.equal(state[1, 0], before[1, 1])


# ---------------------------------------------------------------------------------------------
# gated linear attention
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,C,R,tau", [(1, 30, 16, 4.0), (9, 130, 1, 1.0), (40, 64, 70, 16.0), (300, 7, 33, 0.5)])
def test_decay_from_a_low_rank_map(T, C, R, tau):
    low = _rand(T, R + 5, seed=T, scale=2.0).float()
    w, b = _rand(C, R, seed=1).float(), _rand(C, seed=2, scale=3.0).float()
    b[0], b[C // 2] = 90.0, -90.0                      # a decay of one, and one that is (nearly) zero
    alpha = torch.full((T, C), float("nan"), device=DEV)
    _k().low_rank_decay(alpha, low.to(DEV)[:, 3:3 + R], w.to(DEV), b.to(DEV), tau)
    want = plain.key_decay(low.double()[:, 3:3 + R] @ w.double().T + b.double(), tau)
    got = alpha.double().cpu()
    assert ((got - want).abs() <= 2e-5 * want + 1e-30).all()


def _scan_steps(H, d, dv, lens, cuts, seed, alpha_of=None, qkv_of=None):
    k = _k()
    qkv = [qkv_of(i, n) if qkv_of else _rand(n, H * (2 * d + dv), seed=seed + i).float() for i, n in enumerate(lens)]
    al = [alpha_of(i, n) if alpha_of else torch.sigmoid(_rand(n, H * d, seed=seed + 50 + i, scale=2.0)).float()
          for i, n in enumerate(lens)]
    slots = [len(lens) - i for i in range(len(lens))]
    state = torch.full((len(lens) + 1, H, d, dv), 7.0, device=DEV)
    for s in slots:
        state[s].zero_()
    at, outs = [0] * len(lens), [[] for _ in lens]
    pad = 4                                              # further columns of the rows
    for step in cuts:
        rows = [(r, at[r], at[r] + n) for r, n in step]
        _, q_start, sl = _batch([n for _, n in step], [slots[r] for r, _ in step])
        T = sum(n for _, n in step)
        proj = torch.full((T, H * (2 * d + dv) + pad), float("nan"), device=DEV)
        proj[:, :H * (2 * d + dv)] = torch.cat([qkv[r][a:b] for r, a, b in rows]).to(DEV)
        o = torch.full((T, H * dv), float("nan"), device=DEV)
        k.linear_scan(o, proj, torch.cat([al[r][a:b] for r, a, b in rows]).to(DEV), state, q_start, sl, len(step), H, d, dv, d ** -0.5)
        o = o.double().cpu()
        i = 0
        for r, a, b in rows:
            outs[r].append(o[i:i + b - a])
            i += b - a
            at[r] = b
    want = []
    for x, a, n in zip(qkv, al, lens):
        q, kk, v = x.double().split([H * d, H * d, H * dv], dim=1)
        o, S = plain.linear_recurrence(q.reshape(n, H, d) * d ** -0.5, kk.reshape(n, H, d), v.reshape(n, H, dv),
                                       a.double().view(n, H, d))
        want.append((o.reshape(n, H * dv), S))
    for r, s in enumerate(slots):
        assert (state[s].double().cpu() - want[r][1]).abs().max() <= 2e-5 * (1 + want[r][1].abs().max())
    free = [s for s in range(len(lens) + 1) if s not in slots]
    assert all((state[s] == 7.0).all() for s in free), "a slot of no request was written"
    return [torch.cat(o) for o in outs], [w[0] for w in want]


@pytest.mark.parametrize("H,d,dv", [(3, 10, 14), (1, 7, 5), (2, 48, 40), (4, 32, 16), (1, 16, 300), (2, 130, 64), (1, 300, 20),
                                    (8, 64, 128), (2, 1, 1)])
def test_scan_however_the_tokens_are_cut(H, d, dv):
    lens = [70, 33, 5]
    for cuts in ([[(0, 70), (1, 33), (2, 5)]],
                 [[(0, 2), (1, 17)], [(2, 3), (0, 31)], [(0, 1), (1, 1), (2, 1)], [(1, 15), (0, 36), (2, 1)]],
                 [[(0, 60), (1, 30)]] + [[(0, 1), (2, 1)]] * 5 + [[(0, 1), (1, 1)]] * 3 + [[(0, 1)]] * 2):
        got, want = _scan_steps(H, d, dv, lens, cuts, seed=H + d)
        for g, w in zip(got, want):
            assert (g - w).abs().max() <= 2e-5 * (1 + w.abs().max())


def test_a_token_written_long_ago_is_read_through_decays_of_one():
    """One token writes a key that nothing else uses; hundreds of tokens (and many tiles) later a query for it brings
    its value back whole, while a second channel whose decay is one half has forgotten it."""
    H, d, dv, n = 1, 12, 8, 500

    def qkv(i, T):
        x = torch.zeros(T, 2 * d + dv)
        x[:, :d] = _rand(T, d, seed=4).float()
        x[:, 0] = x[:, 1] = 0
        x[:, d + 2:2 * d] = _rand(T, d - 2, seed=5).float()
        x[:, 2 * d:] = _rand(T, dv, seed=6).float()
        x[3, d], x[3, d + 1] = 2.0, 2.0                  # the planted write, on channels 0 and 1
        x[n - 2, :d] = 0
        x[n - 2, 0] = d ** 0.5                           # asks channel 0
        x[n - 1, :d] = 0
        x[n - 1, 1] = d ** 0.5                           # asks channel 1
        return x

    def alpha(i, T):
        a = torch.full((T, d), 0.9)
        a[:, 0], a[:, 1] = 1.0, 0.5
        return a

    for cuts in ([[(0, n)]], [[(0, 5)], [(0, n - 12)]] + [[(0, 1)]] * 7):
        got, want = _scan_steps(H, d, dv, [n], cuts, seed=0, alpha_of=alpha, qkv_of=qkv)
        v3 = qkv(0, n)[3, 2 * d:].double()
        assert (got[0][n - 2] - 2.0 * v3).abs().max() < 1e-5 and got[0][n - 1].abs().max() < 1e-6
        assert (got[0] - want[0]).abs().max() <= 2e-5 * (1 + want[0].abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dv", [(3, 14), (2, 64), (1, 200), (1, 700)])
def test_norm_per_head_and_silu_gate(dtype, H, dv):
    T, eps = 11, 1e-5
    o, row, w = _rand(T, H * dv, seed=1).float(), _rand(T, H * dv + 7, seed=2, scale=2.0).float(), (1 + _rand(dv, seed=3, scale=0.3)).float()
    out = torch.full((T, H * dv), float("nan"), dtype=dtype, device=DEV)
    _k().gated_head_norm(out, o.to(DEV), row.to(DEV), 7, w.to(DEV), dv, eps, gate_after=True, silu_gate=True)
    g = row.double()[:, 7:]
    want = plain.rms_norm(o.double().view(T, H, dv), w.double(), eps).reshape(T, H * dv) * g * torch.sigmoid(g)
    assert (out.double().cpu() - want).abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2) * (1 + want.abs().max())


# ---------------------------------------------------------------------------------------------
# the router and the experts
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,scale", [(5, 2, 1.5), (12, 4, 2.5), (1, 1, 1.0), (7, 7, 0.8), (64, 6, 3.0), (33, 1, 2.0)])
@pytest.mark.parametrize("gated", [False, True])
def test_softmax_router_chooses_as_plain(dtype, E, top, scale, gated):
    T, K = 37, 52
    h = _rand(T, K, seed=E).to(dtype)
    w = _rand(E + gated, K, seed=E + 1, scale=0.4).float()
    h[7] *= 40.0                                                     # logits far apart: most scores underflow
    choice = torch.full((T, top), -7, dtype=torch.int32, device=DEV)
    weight = torch.full((T, top), float("nan"), dtype=torch.float32, device=DEV)
    gate = torch.full((T,), float("nan"), dtype=torch.float32, device=DEV) if gated else None
    req = torch.zeros(T, dtype=torch.int32)
    req[5] = -1                                                      # a padding token takes part in nothing
    _k().expert_router(choice, weight, h.to(DEV), w.to(DEV), None, req.to(DEV), top, renormalize=True, softmax=True,
                       renormalize_eps=1e-20, weight_scale=scale, gate=gate)
    idx, wt = plain.route(h.double(), w.double()[:E], top, scale)
    got_i, got_w = choice.cpu(), weight.double().cpu()
    for t in range(T):
        if t == 5:
            assert got_w[t].abs().max() == 0
            continue
        if t != 7:
            assert got_i[t].tolist() == idx[t].tolist(), t
        assert (got_w[t] - wt[t]).abs().max() < 2e-5 * scale
    if gated:
        want = torch.sigmoid(h.double() @ w.double()[E])
        keep = [t for t in range(T) if t != 5]
        assert (gate.double().cpu()[keep] - want[keep]).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 3, 70])
@pytest.mark.parametrize("E,top,shared", [(6, 2, 16), (1, 1, 24), (5, 5, 20), (4, 3, None)])
def test_routed_experts_part_equals_plain(dtype, T, E, top, shared):
    """The part alone, few tokens (in bfloat16 two dense products over all experts and the shared one) and many
    (grouped products, per-expert library products), with a padding token, against the plain mixture."""
    from xinfer_b200.config.plan import FeedForwardSpec, RoutedExpertsSpec
    from xinfer_b200.parts import Workspace, build_part
    from xinfer_b200.parts.base import StepContext
    H, Fi, scale = 48, 24, 1.7
    mlp = dict(kind="moe", expert=dict(ff=Fi), router=dict(experts=E, top=top, scale=scale))
    names = [f"m.e{e}.{n}" for e in range(E) for n in ("gate", "up", "down")]
    if shared:
        mlp["shared"] = dict(ff=shared)
        names += ["m.shared.gate", "m.shared.up", "m.shared.down"]
    w = {}
    for i, n in enumerate(names):
        ff = shared if "shared" in n else Fi
        w[n] = (_rand(*((H, ff) if n.endswith("down") else (ff, H)), seed=100 + i, scale=0.2)).to(dtype).double()
    w["m.router"] = _rand(E, H, seed=7, scale=0.3).to(dtype).double()
    w["m.shared.sg"] = _rand(1, H, seed=8, scale=0.3).to(dtype).double()

    class Store:
        def get(self, name, device, dt, operand=False, columns=None):
            return w[name].to(dt).to(device)

    sh = FeedForwardSpec(kind="swiglu", hidden=H, intermediate=shared, activation="silu", names=("gate", "up", "down")) if shared else None
    spec = RoutedExpertsSpec(kind="routed_experts", hidden=H, intermediate=Fi, experts=E, top=top, correction=False, renormalize=True,
                             score="softmax", renormalize_eps=1e-20, weight_scale=scale, shared=sh,
                             shared_gate="shared.sg" if shared else None)
    part = build_part("feed_forward", spec, "m.", dtype, DEV)
    part.load(Store())
    x = _rand(T, H, seed=T).to(dtype)
    req = torch.zeros(T, dtype=torch.int32)
    if T > 1:
        req[1] = -1
    ctx = StepContext(dtype=dtype, device=torch.device(DEV), num_tokens=T, num_entries=1, token_ids=_i32([0] * T),
                      positions=_i32(list(range(T))), req_of_token=req.to(DEV), q_start=_i32([0, T]), start_pos=_i32([0]),
                      slots=_i32([0]), logit_rows=_i32([0]), num_logit_rows=0, tables=[], strides=[], err=_err(),
                      workspace=Workspace(DEV), branch_dtype=torch.float32)
    want = plain.routed_experts(x.double(), w, "m.", mlp)
    keep = [t for t in range(T) if t != 1]
    tol = (2e-5 if dtype == torch.float32 else 4e-2) * (1 + want.abs().max())
    out = part.forward(x.to(DEV), ctx).double().cpu()
    assert int(ctx.err.item()) == 0
    assert (out[keep] - want[keep]).abs().max() <= tol
    if dtype == torch.bfloat16 and T > 32:
        # the form of large prompt steps: every expert's rows through the library's product
        from xinfer_b200.parts import routed_experts as form
        before, floor = _k().launch_counts().get("expert_gather", 0), form.LIBRARY_FROM_FLOP_PER_CALL
        form.LIBRARY_FROM_FLOP_PER_CALL = 0.0
        try:
            again = part.forward(x.to(DEV), ctx).double().cpu()
        finally:
            form.LIBRARY_FROM_FLOP_PER_CALL = floor
        assert _k().launch_counts().get("expert_gather", 0) == before + 1
        assert (again[keep] - want[keep]).abs().max() <= tol


# ---------------------------------------------------------------------------------------------
# attention over a cached latent
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank,rd,nq", [(14, 4, 18), (48, 16, 32), (40, 6, 300)])
def test_latent_rows_and_the_queries_own_latent(dtype, rank, rd, nq):
    T, ps, eps = 21, 8, 1e-5
    row = _rand(T, nq + rank + rd + 3, seed=rank, scale=2.0).to(dtype)
    wn, qn = (1 + _rand(rank, seed=1, scale=0.3)).float(), (1 + _rand(nq, seed=2, scale=0.3)).float()
    rot = dict(dims=rd - 2, base=70.0, scaling=dict(factor=3.0, original=64, fast=4.0, slow=0.5))
    f, mag = plain.yarn_frequencies(rot["dims"], rot["base"], rot["scaling"])
    pos = [5 + i for i in range(T)]
    pages = (max(pos) + ps) // ps
    table = torch.randperm(pages + 2, generator=torch.Generator().manual_seed(5))[:pages].to(torch.int32)
    cache = torch.full((pages + 2, ps, rank + rd), float("nan"), dtype=dtype, device=DEV)
    cq = torch.full((T, nq), float("nan"), dtype=dtype, device=DEV)
    err = _err()
    _k().latent_prepare(None, cache, row.to(DEV), 0, nq, None, wn.to(DEV), f.float().to(DEV), _i32(pos), _i32([0] * T),
                        table.to(DEV).view(1, -1), pages, 0, 0, rd, rank, rot["dims"], eps, mag, err, query_latent=(cq, 0, qn.to(DEV)))
    assert int(err.item()) == 0
    x = row.double()
    want = plain.rms_norm(x[:, :nq], qn.double(), eps)
    assert (cq.double().cpu() - want).abs().max() <= _tol(dtype) * (1 + want.abs().max())
    c = plain.rms_norm(x[:, nq:nq + rank], wn.double(), eps)
    kr = plain.rotate_neighbours(x[:, None, nq + rank:nq + rank + rd], torch.tensor(pos), rot)[:, 0]
    for i, p in enumerate(pos):
        got = cache[int(table[p // ps]), p % ps].double().cpu()
        assert (got - torch.cat([c[i], kr[i]])).abs().max() <= _tol(dtype) * (1 + x.abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_query_rows_are_zero_where_the_cached_rows_are_not_this_layers(dtype):
    T, nh, d, rank, tail = 5, 3, 6, 12, 4
    q_abs = torch.full((T, nh, rank + tail), float("nan"), dtype=dtype, device=DEV)
    q_abs[:, :, :rank] = 1.5
    cache = torch.zeros(2, 8, rank + tail, dtype=dtype, device=DEV)
    proj = torch.zeros(T, nh * d, dtype=dtype, device=DEV)
    err = _err()
    _k().latent_prepare(q_abs, cache, proj, 0, -1, None, None, None, _i32([0] * T), _i32([0] * T), _i32([[0]]), 1, nh, d, 0, rank, 0,
                        1e-6, 1.0, err, tail=tail)
    assert (q_abs[:, :, :rank] == 1.5).all() and (q_abs[:, :, rank:] == 0).all() and int(err.item()) == 0


class _Ctx:
    """The fields of a step context that the latent attention reads, for requests whose rows already lie in pages (in
    a scrambled order) and whose last ``len - start`` tokens are this step's queries."""

    def __init__(self, rows, starts, ps, dtype, seed):
        from xinfer_b200.parts import Workspace
        lens = [r.shape[0] for r in rows]
        need = [(n + ps - 1) // ps for n in lens]
        total = sum(need) + 3
        order = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
        pages = torch.full((total, ps, rows[0].shape[1]), float("nan"), dtype=dtype)
        self.stride = max(need) + 2
        table = torch.full((len(rows), self.stride), -1, dtype=torch.int32)
        at = 0
        for b, r in enumerate(rows):
            for p in range(need[b]):
                table[b, p] = order[at]
                n = min(ps, lens[b] - p * ps)
                pages[order[at], :n] = r[p * ps:p * ps + n].to(dtype)
                at += 1
        counts = [n - s for n, s in zip(lens, starts)]
        self.bounds = np.concatenate([[0], np.cumsum(counts)]).tolist()
        self.pages, self.table = pages.to(DEV), table.to(DEV)
        self.q_start, self.start_pos = _i32(self.bounds), _i32(starts)
        self.num_entries, self.num_tokens = len(rows), int(self.bounds[-1])
        self.positions = _i32([s + i for s, c in zip(starts, counts) for i in range(c)])
        self.req_of_token = _i32([b for b, c in enumerate(counts) for _ in range(c)])
        self.all_single = all(c == 1 for c in counts)
        self.fixed_shapes = False
        self.max_context = max(lens)
        self.workspace = Workspace(DEV)
        self.err = _err()


def _attend(qs, rows, starts, rank, scale, ps, dtype, window, tiled=True, seed=0):
    """qs: queries in the latent space per request [n, H, dk]; rows: what the requests cached [n, dk]."""
    from xinfer_b200.parts import latent_attention as la
    ctx = _Ctx(rows, starts, ps, dtype, seed)
    q = torch.cat([q[s:] for q, s in zip(qs, starts)]).to(dtype).to(DEV).contiguous()
    out = torch.full((q.shape[0], q.shape[1], rank), float("nan"), dtype=dtype, device=DEV)
    la.USE_TENSOR_CORES = tiled
    try:
        la.latent_attend(out, q, ctx.pages, ctx, ctx.table, ctx.stride, ps, window, scale, None)
    finally:
        la.USE_TENSOR_CORES = True
    torch.cuda.synchronize()
    assert int(ctx.err.item()) == 0
    res = out.double().cpu()
    return [res[a:b] for a, b in zip(ctx.bounds[:-1], ctx.bounds[1:])]


def _attend_plain(q, row, rank, scale, window):
    n, H = q.shape[:2]
    k = row[:, None, :].expand(n, H, row.shape[1])
    return plain.softmax_heads(q, k, k[..., :rank], plain.causal_mask(n, window), scale)


# (dtype, tiled): float32 on the plain kernel, bfloat16 on the tensor-core kernel and on the plain one
FORMS = [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)]


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("H,rank,rest,ps", [(3, 20, 0, 8), (8, 64, 0, 16), (4, 128, 0, 16), (2, 48, 16, 32), (1, 256, 0, 16)])
@pytest.mark.parametrize("window", [None, 50, 1])
def test_attention_of_unequal_entries_equals_plain(dtype, tiled, H, rank, rest, ps, window):
    """Prompt portions of several lengths, one that continues a cached prefix, single tokens, all in one batch; rows
    with and without channels behind the latent."""
    lens, starts = [150, 61, 200, 97, 1], [0, 40, 199, 96, 0]
    rows = [_rand(n, rank + rest, seed=10 * b).to(dtype).double() for b, n in enumerate(lens)]
    qs = [(_rand(n, H, rank + rest, seed=10 * b + 1) * 1.5).to(dtype).double() for b, n in enumerate(lens)]
    got = _attend(qs, rows, starts, rank, rank ** -0.5, ps, dtype, window, tiled, seed=3)
    for q, r, s, o in zip(qs, rows, starts, got):
        ref = _attend_plain(q, r, rank, rank ** -0.5, window)[s:]
        assert (o - ref).abs().max() <= _tol(dtype) * (1 + ref.abs().max())


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("window", [48, 64, 2, 200, 11, 130])
def test_window_edges(dtype, tiled, decode, window):
    """One row is made to stand out for the last query: inside the window it decides the output, one token further
    back it must not be seen."""
    H, rank, ps, n = 4, 32, 16, 260
    for j, inside in [(n - window, True), (n - window - 1, False), (n - 1, True)]:
        row = _rand(n, rank, seed=6).to(dtype).double()
        q = _rand(n, H, rank, seed=7).to(dtype).double()
        q[-1] = row[j] * 2.0
        q = q.to(dtype).double()
        start = n - 1 if decode else n - 9
        got = _attend([q], [row], [start], rank, 1.0, ps, dtype, window, tiled)[0]
        ref = _attend_plain(q, row, rank, 1.0, window)[start:]
        assert (got - ref).abs().max() <= _tol(dtype) * (1 + ref.abs().max())
        carried = (got[-1, 0] - row[j]).abs().max() < 8e-2 * (1 + row.abs().max())
        assert bool(carried) == inside, (j, inside)


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("where", ["first", "second", "page_end", "page_start", "tile_end", "tile_start", "far", "previous"])
def test_one_planted_row_decides_the_output(dtype, tiled, where, decode):
    H, rank, ps, n = 8, 64, 16, 600
    j = {"first": 0, "second": 1, "page_end": 31, "page_start": 32, "tile_end": 63, "tile_start": 64, "far": n - 517,
         "previous": n - 2}[where]
    row = _rand(n, rank, seed=99).to(dtype).double()
    q = _rand(n, H, rank, seed=98).to(dtype).double()
    q[-1] = row[j]
    start = n - 1 if decode else n - 37
    got = _attend([q], [row], [start], rank, 0.8, ps, dtype, None, tiled)[0]
    ref = _attend_plain(q, row, rank, 0.8, None)[start:]
    assert (got - ref).abs().max() <= _tol(dtype) * (1 + ref.abs().max())
    assert (got[-1, H - 1] - row[j]).abs().max() < 8e-2 * (1 + row.abs().max()), "the planted row must carry the output"


# ---------------------------------------------------------------------------------------------
# whole models: every way of cutting, pages and slots used again, layer by layer, generation
# ---------------------------------------------------------------------------------------------
LENGTHS = {"N1": [70, 45, 130, 33], "N2": [97, 41, 260, 150], "N3": [170, 1, 75, 58], "N4": [90, 2, 51, 140]}


def _tolerance(dtype, ref, cfg=None, w=None, p=None, routes=None):
    """float32: a small share of the logits' spread (the engine's float32 against float64).  bfloat16: three
    times what rounding alone causes - the largest row error of the plain run that rounds activations to
    bfloat16 where an engine stores them (along the same experts: another choice is no rounding error)."""
    spread = max(float(np.std(ref)), 1e-3)
    if dtype == "float32":
        return 3e-5 * spread
    rounded = plain.forward(cfg, w, p, round_to=torch.bfloat16, routes=routes, slack=float("inf")).numpy()
    return max(3.0 * max(row_error(rounded[i], ref[i]) for i in range(len(p))), 1e-3 * spread)


def _store(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


@pytest.mark.parametrize("name", sorted(TINY_N))
def test_every_way_of_cutting_gives_the_plain_logits_in_float32_through_the_replay_program(name, tmp_path):
    dtype = "float32"
    folder = make_folder(str(tmp_path / "model"), name, _store(dtype))
    ps = prompts(name, LENGTHS[name])
    tb = build_all_modes(ps, seed=len(name))
    out = run_trace(folder, dtype, tb.steps, str(tmp_path / "out"), max_tokens=tb.peak, page_size=TINY_N[name][2],
                    max_num_seqs=4)
    cfg, w = plain.load_folder(folder)
    ref = [plain.forward(cfg, w, p).numpy() for p in ps]
    tol = [_tolerance(dtype, r, cfg, w, p) for r, p in zip(ref, ps)]
    seen = {}
    for step, rows in tb.rows.items():
        got = out[step]
        assert got.shape[0] == len(rows)
        for r, ((mode, i), pos) in enumerate(rows):
            e = row_error(got[r], ref[i][pos])
            assert e <= tol[i], (f"{name} {mode}: request {i} position {pos} (step {step}) differs by {e:.3g} "
                                 f"> {tol[i]:.3g}: the first wrong token of this mode")
            seen.setdefault((mode, i), set()).add(pos)
    for mode in ("whole", "tail", "portions", "mixed"):
        for i, p in enumerate(ps):
            assert sorted(seen[(mode, i)]) == list(range(len(p))), (mode, i)


def _check_trace(name, dtype, runner, tb, ps, cfg, w):
    """Replays the trace and compares every wanted row with the plain run of its request.  An engine that rounds
    activations may decide a router's close call the other way, after which the request is another computation:
    the engine's choices are recorded, checked to differ from the plain ones by close calls only, and followed by
    the plain run (in float32 nothing is close: the slack is a rounding error's)."""
    L = len(cfg["layers"])
    moe_runs = [i for i in range(L) if (cfg["layers"][i].get("mlp") or {}).get("kind") == "moe"]
    out, routes = replay_with_routes(runner, tb.steps, moe_runs)
    slack = 1e-4 if dtype == "float32" else 0.5          # (a router's logits are a few units apart)
    ref, tol = {}, {}         # per request id of the trace: the plain logits along the engine's routes

    def plain_of(rid, i):
        if rid not in ref:
            given = [routes[rid].get(run) for run in range(L)]
            if all(g is None for g in given):
                given = None
            ref[rid] = plain.forward(cfg, w, ps[i], routes=given, slack=slack).numpy()
            tol[rid] = _tolerance(dtype, ref[rid], cfg, w, ps[i], given)
        return ref[rid], tol[rid]

    seen, worst = {}, {}
    for step, rows in tb.rows.items():
        got = out[step]
        assert got.shape[0] == len(rows)
        assert np.isfinite(got).all(), f"step {step} read a stale page"
        rid_of_row = [e["id"] for e in tb.steps[step]["entries"] for _ in e["want"]]
        for r, ((mode, i), pos) in enumerate(rows):
            want, t = plain_of(rid_of_row[r], i)
            e = row_error(got[r], want[pos])
            worst[mode] = max(worst.get(mode, 0.0), e / t)
            assert e <= t, (f"{name} {dtype} {mode}: request {i} position {pos} (step {step}) differs by {e:.3g} "
                            f"> {t:.3g}: the first wrong token of this mode")
            seen.setdefault((mode, i), set()).add(pos)
    for mode in ("whole", "tail", "portions", "mixed"):
        for i, p in enumerate(ps):
            assert sorted(seen[(mode, i)]) == list(range(len(p))), (mode, i)
    return worst


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY_N))
def test_every_way_of_cutting_gives_the_plain_logits(name, dtype, tmp_path):
    """Every request whole, with its tail token by token, in portions, and four at a time over a pool of the live
    requests' size, against the plain run."""
    from xinfer_b200.engine.runner import ModelRunner
    folder = make_folder(str(tmp_path / "model"), name, _store(dtype))
    ps = prompts(name, LENGTHS[name])
    tb = build_all_modes(ps, seed=len(name))
    page = TINY_N[name][2]
    runner = ModelRunner(folder, dtype, block_size=page, num_blocks=(tb.peak + page - 1) // page, max_num_seqs=4)
    cfg, w = plain.load_folder(folder)
    worst = _check_trace(name, dtype, runner, tb, ps, cfg, w)
    print(name, dtype, "worst error / tolerance per mode:", {k: f"{v:.3g}" for k, v in worst.items()})


@pytest.mark.parametrize("name,dtype", [("N1", "float32"), ("N2", "bfloat16"), ("N3", "bfloat16"), ("N4", "float32")])
def test_freed_pages_and_slots_are_used_again_and_nothing_stale_is_read(name, dtype, tmp_path):
    """Pages that go back to the pool are filled with NaN before the next step (also the pages that windows give
    back while a request runs), and every state row starts out as junk.  Eight requests pass through four slots and a
    pool of the live requests' size: the logits stay the plain ones and stay finite."""
    from xinfer_b200.engine.runner import ModelRunner
    folder = make_folder(str(tmp_path / "model"), name, _store(dtype))
    ps = prompts(name, LENGTHS[name])
    tb = build_all_modes(ps, seed=3)
    page = TINY_N[name][2]
    runner = ModelRunner(folder, dtype, block_size=page, num_blocks=(tb.peak + page - 1) // page, max_num_seqs=4,
                         poison_freed_pages=True)
    for t in runner.state.tables.values():
        t.fill_(1e4)
    cfg, w = plain.load_folder(folder)
    _check_trace(name, dtype, runner, tb, ps, cfg, w)
    assert runner.pages_poisoned > runner.num_blocks


@pytest.mark.parametrize("name", sorted(TINY_N))
def test_layers_one_by_one_in_float32(name, tmp_path):
    """The residual stream after every layer against the plain one, a prompt in two portions."""
    from xinfer_b200.engine.runner import ModelRunner, StepInput
    from xinfer_b200.parts.block import Block
    folder = make_folder(str(tmp_path / "model"), name, torch.float32)
    cfg, w = plain.load_folder(folder)
    p = prompts(name, [29])[0]
    want = []
    plain.forward(cfg, w, p, streams=want)
    rec, orig = [], Block.forward

    def spy(self, stream, ctx, cache, state, writes_cache):
        out = orig(self, stream, ctx, cache, state, writes_cache)
        out.settle(ctx)
        rec.append(out.x.double().cpu())
        return out

    Block.forward = spy
    try:
        runner = ModelRunner(folder, "float32", block_size=8, num_blocks=64, max_num_seqs=2)
        slot = runner.open_request()
        runner.step([StepInput(slot, p[:11], [])])
        first = list(rec)
        rec.clear()
        runner.step([StepInput(slot, p[11:], [])])
        runner.check_errors()
    finally:
        Block.forward = orig
    assert len(rec) == len(first) == len(want)
    for i, (a, b, ref) in enumerate(zip(first, rec, want)):
        got = torch.cat([a[:11], b[: len(p) - 11]])
        assert got.dtype == F64 and (got - ref).abs().max() <= 2e-5 * (1 + ref.abs().max()), f"layer {i}"


def test_the_stream_is_float32_and_the_fused_and_fast_kernels_run_in_bfloat16(tmp_path):
    from xinfer_b200 import kernels
    from xinfer_b200.engine.runner import ModelRunner, StepInput
    folder = make_folder(str(tmp_path / "model"), "N2", torch.bfloat16)
    runner = ModelRunner(folder, "bfloat16", block_size=16, num_blocks=64, max_num_seqs=2)
    assert runner.model.stream_dtype == torch.float32 and runner.model.dtype == torch.bfloat16
    assert runner.model.graph_safe()
    slot = runner.open_request()

    def launched(tokens, want):
        before = dict(kernels.launch_counts())
        runner.step([StepInput(slot, tokens, want)])
        runner.check_errors()
        return {k: n - before.get(k, 0) for k, n in kernels.launch_counts().items() if n > before.get(k, 0)}

    first, then = launched(list(range(40)), [39]), launched([5], [0])
    for used in (first, then):
        assert "attn_latent_mma" in used and "attention_plain" not in used, sorted(used)
        # the stream's sums: one per feed-forward with the convolution (or the final norm) behind it, one per mixer with
        # the feed-forward behind it; no addition kernel, no norm kernel of its own
        assert used["stream_conv"] == 5 and used["rms_chain"] == 5 and "add_f32" not in used and "rmsnorm_f32" not in used, used
    # one token per request: the convolution's inputs are kept in the same launch, the shared expert runs with the others
    assert first["conv_state"] == 5 and "conv_state" not in then
    assert "expert_gemm_mma" in first and "expert_combine" in first
    assert then["expert_select_gate"] == 3 and "expert_combine" not in then


def test_layers_that_share_rows_own_no_cache_and_widths_count_the_inner_parts(tmp_path):
    from xinfer_b200.engine.runner import ModelRunner
    folder = make_folder(str(tmp_path / "model"), "N2", torch.bfloat16)
    runner = ModelRunner(folder, "bfloat16", block_size=16, num_blocks=16, max_num_seqs=2)
    caches = runner.layer_caches
    assert [c is None for c in caches] == [False, True, False, True, True]
    assert caches[0]["latent"].shape[-1] == 64 and caches[2]["latent"].shape[-1] == 64 and caches[0].group != caches[2].group
    cfg, w = plain.load_folder(folder)
    # every tensor once: bfloat16 operands, float32 norms, filters, routers and the second half of the decay's map
    assert runner.model.weight_bytes() >= 2 * sum(t.numel() for t in w.values())


def _engine(folder, dtype, page, **kw):
    from xinfer_b200 import Engine, EngineConfig
    opts = dict(weight_path=folder, block_size=page, num_blocks=96, max_num_seqs=4, max_num_batched_tokens=64,
                prefill_chunk_size=16, disable_cuda_graph=True, max_model_len=1024)
    opts.update(kw)
    return Engine(EngineConfig(**opts), dtype)


@pytest.mark.parametrize("name", ["N1", "N3", "N4"])
def test_greedy_generation_in_float32_equals_plain(name, tmp_path):
    from xinfer_b200 import SamplingParams
    folder = make_folder(str(tmp_path / "model"), name, torch.float32)
    cfg, w = plain.load_folder(folder)
    ps = prompts(name, [1, 5, 23, 40, 9, 17])       # six requests over four slots, prompts in portions of 16
    eng = _engine(folder, "f32", TINY_N[name][2])
    outs = eng.generate_sync(SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True), ps)
    for p, o in zip(ps, outs):
        assert o.decode_output == plain.greedy(cfg, w, p, 12)


@pytest.mark.parametrize("graphs", [False, True], ids=["launched", "cuda_graph"])
@pytest.mark.parametrize("name", ["N2", "N4"])
def test_long_greedy_decoding_in_bfloat16_follows_the_plain_logits(name, graphs, tmp_path):
    """Each generated token is checked against the plain logits of the sequence the engine produced (bfloat16
    may flip a near-tie): it must be the best token up to the drift.  Long enough for many pages per request and for
    windows to pass over decoded tokens."""
    from xinfer_b200 import SamplingParams
    folder = make_folder(str(tmp_path / "model"), name, torch.bfloat16)
    cfg, w = plain.load_folder(folder)
    ps = prompts(name, [3, 30, 61])
    eng = _engine(folder, "bf16", TINY_N[name][2], disable_cuda_graph=not graphs)
    outs = eng.generate_sync(SamplingParams(max_tokens=150, ignore_eos=True), ps)
    assert eng.runner.last_used_graph == graphs
    for p, o in zip(ps, outs):
        assert o.decoded_length == 150
        seq = p + o.decode_output
        ref = plain.forward(cfg, w, seq)
        slack = 2 * 3.0 * float((plain.forward(cfg, w, seq, round_to=torch.bfloat16) - ref).abs().max())
        for i, tok in enumerate(o.decode_output):
            row = ref[len(p) + i - 1]
            assert row[tok] >= row.max() - slack, (i, tok)


def test_command_line_writes_a_random_folder_and_generates_from_it(tmp_path, capsys):
    """The command line end to end: a folder from a configuration and a seed, then generation from given ids (equal
    to the plain continuation in float32) and from a seeded prompt of a given length."""
    import json
    from xinfer_b200.cli import main
    config = tmp_path / "config.json"
    config.write_text(json.dumps(TINY_N["N1"][0]))
    folder = str(tmp_path / "model")
    assert main(["--random", str(config), "--seed", "4", "--m", folder, "--store-dtype", "f32"]) == 0
    cfg, w = plain.load_folder(folder)
    capsys.readouterr()
    assert main(["--m", folder, "--dtype", "f32", "--prompts", "5,6,7|9,10", "--max-tokens", "4", "--ignore-eos",
                 "--disable-cuda-graph", "--num-blocks", "32"]) == 0
    out = capsys.readouterr().out
    assert ",".join(str(t) for t in plain.greedy(cfg, w, [5, 6, 7], 4)) in out and "Decoded tokens: 8" in out
    assert main(["--m", folder, "--prompt-len", "21", "--batch", "3", "--max-tokens", "5", "--ignore-eos", "--num-blocks", "32",
                 "--seed", "1"]) == 0
    assert "Decoded tokens: 15" in capsys.readouterr().out
