"""The Dalalix decoder on the GPU against the plain implementation (plain_dalalix.py): every mechanism alone through its
kernel, then whole models through the step function, the replay program and the generation entry point - whole prompts,
token-by-token decoding, portions down to two tokens, unequal batches, pages and slots that are used again, keys far back
and at the edges of windows, kept ranges, pages and tiles, the first tokens of a sequence."""
import numpy as np
import pytest
import torch

import plain_dalalix as plain
from dalalix_models import TINY_D, make_folder, prompts
from helpers import build_all_modes, replay_with_routes, row_error, run_trace

pytestmark = pytest.mark.gpu

DEV = "cuda:0"


@pytest.fixture(autouse=True)
def _one_thread():
    """The plain implementation works on small matrices: threads would only wait for each other."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


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


# ---------------------------------------------------------------------------------------------
# several residual streams
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,T,W", [(1, 5, 48), (2, 9, 52), (3, 33, 37), (4, 400, 64), (4, 3, 4096), (5, 7, 40), (8, 11, 100), (9, 6, 44),
                                   (32, 4, 130)])
def test_streams_are_mixed_read_and_normed(n, T, W, dtype):
    eps = 1e-5
    X, y = _rand(n, T, W, seed=n), _rand(T, W, seed=n + 1, scale=2.0)
    M, w, r, nw = _rand(n, n, seed=2), _rand(n, seed=3), _rand(n, seed=4), 1 + _rand(W, seed=5, scale=0.3)
    f = lambda t: t.float().to(DEV).contiguous()
    X, y, M, w, r, nw = (t.float().double() for t in (X, y, M, w, r, nw))
    new = plain.write_streams(X, M, w, y)
    scale = 1 + new.abs().max()
    for branch_dtype in (torch.float32, torch.bfloat16):
        yy = y.to(branch_dtype)
        new = plain.write_streams(X, M, w, yy.double())
        u = plain.read_streams(new, r)
        want = plain.rms_norm(u, nw, eps)
        x = f(X.permute(1, 0, 2))
        out = torch.full((T, W), float("nan"), dtype=dtype, device=DEV)
        err = _err()
        _k().stream_mix(out, x, f(r), f(nw), eps, err, branch=yy.to(DEV), mix=f(M), write=f(w), x_out=x)     # in place
        assert (x.double().cpu().permute(1, 0, 2) - new).abs().max() <= 1e-5 * scale
        assert (out.double().cpu() - want).abs().max() <= (2e-5 if dtype == torch.float32 else 1e-2) * (1 + want.abs().max())
        # the same sum without a norm, and the streams alone
        x = f(X.permute(1, 0, 2))
        u32, moved = torch.empty(T, W, device=DEV), torch.full_like(x, float("nan"))
        _k().stream_mix(u32, x, f(r), None, 0.0, err, branch=yy.to(DEV), mix=f(M), write=f(w))
        assert (u32.double().cpu() - u).abs().max() <= 1e-5 * scale * n and torch.equal(x, f(X.permute(1, 0, 2)))
        _k().stream_mix(None, x, None, None, 0.0, err, branch=yy.to(DEV), mix=f(M), write=f(w), x_out=moved)
        assert (moved.double().cpu().permute(1, 0, 2) - new).abs().max() <= 1e-5 * scale
        # the plain sum at gathered rows after the last addition
        rows = [T - 1, 0, T // 2, T // 2]
        out = torch.full((4, W), float("nan"), dtype=dtype, device=DEV)
        _k().stream_mix(out, x, None, f(nw), eps, err, branch=yy.to(DEV), mix=f(M), write=f(w), rows=_i32(rows))
        want = plain.rms_norm(new.sum(0)[rows], nw, eps)
        assert (out.double().cpu() - want).abs().max() <= (3e-5 if dtype == torch.float32 else 1e-2) * (1 + want.abs().max())
        assert int(err.item()) == 0


@pytest.mark.parametrize("n,W", [(3, 40), (4, 64), (7, 37)])
def test_equal_streams_are_read_from_one_copy(n, W):
    T, eps = 13, 1e-6
    x0, y = _rand(T, W, seed=1).float(), _rand(T, W, seed=2).float()
    M, w, r, nw = (_rand(*s, seed=i).float().to(DEV) for i, s in enumerate([(n, n), (n,), (n,), (W,)]))
    X = x0.double()[None].repeat(n, 1, 1)
    x = x0.to(DEV).unsqueeze(1).expand(T, n, W)
    out, err = torch.empty(T, W, device=DEV), _err()
    _k().stream_mix(out, x, r, nw, eps, err)                     # nothing has been written to them yet
    want = plain.rms_norm(plain.read_streams(X, r.double().cpu()), nw.double().cpu(), eps)
    assert (out.double().cpu() - want).abs().max() <= 2e-5 * (1 + want.abs().max())
    dst = torch.full((T, n, W), float("nan"), device=DEV)
    _k().stream_mix(out, x, r, nw, eps, err, branch=y.to(DEV), mix=M, write=w, x_out=dst)
    new = plain.write_streams(X, M.double().cpu(), w.double().cpu(), y.double())
    assert (dst.double().cpu().permute(1, 0, 2) - new).abs().max() <= 1e-5 * (1 + new.abs().max())
    with pytest.raises(_k().KernelError):
        _k().stream_mix(out, x, r, nw, eps, err, branch=y.to(DEV), mix=M, write=w, x_out=x)
    # a row outside the step is reported, not read
    _k().stream_mix(out[:1], x, None, nw, eps, err, rows=_i32([T + 4]))
    assert int(err.item()) == _k().ERR_BAD_ROW


# ---------------------------------------------------------------------------------------------
# queries, keys and values: convolution, value norm, biases, rotation of halves
# ---------------------------------------------------------------------------------------------
def _prepare_steps(H, G, d, dv, K, lens, cuts, dtype, seed, value_eps=1e-5, ps=8, extra=5):
    """Runs requests through the prepare kernel in steps (``cuts``: lists of (request, tokens)); returns per request (q,
    k, v) as the kernel left them and the convolved rows as the plain functions give them."""
    k_ = _k()
    C = (H + G) * d + G * dv
    rows = [_rand(n, C, seed=seed + i).to(dtype) for i, n in enumerate(lens)]
    taps = _rand(C, K, seed=seed + 90, scale=0.6).float()
    R = len(lens)
    slots = [R - i for i in range(R)]
    state = torch.full((R + 1, max(K - 1, 1), C), 3.0, dtype=dtype, device=DEV)
    for s in slots:
        state[s].zero_()
    per = (max(lens) + ps - 1) // ps
    order = torch.randperm(R * per, generator=torch.Generator().manual_seed(seed)).tolist()
    tables = [order[i * per:(i + 1) * per] for i in range(R)]
    kc = torch.full((R * per, G, ps, d), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((R * per, G, ps, dv), float("nan"), dtype=dtype, device=DEV)
    at, qs = [0] * R, [[] for _ in lens]
    err = _err()
    for step in cuts:
        parts = [(r, at[r], at[r] + n) for r, n in step]
        T = sum(n for _, n in step)
        qkv = torch.full((T, C + extra), 9.0, dtype=dtype, device=DEV)
        qkv[:, :C] = torch.cat([rows[r][a:b] for r, a, b in parts]).to(DEV)
        q_start = np.concatenate([[0], np.cumsum([n for _, n in step])]).tolist()
        pos = [p for _, a, b in parts for p in range(a, b)]
        req = [j for j, (_, a, b) in enumerate(parts) for _ in range(a, b)]
        q = torch.full((T, H, d), float("nan"), dtype=dtype, device=DEV)
        k_.qkv_prepare(q, kc, vc, qkv, None, None, None, _i32(pos), _i32(req), _i32([tables[r] for r, _ in step]), per, H, G, d, dv, 0,
                       False, 0, 1e-6, True, err, row_len=C + extra, value_eps=value_eps,
                       conv=(taps.t().contiguous().to(DEV), state if K > 1 else None, _i32(q_start), _i32([slots[r] for r, _ in step]),
                             all(n == 1 for _, n in step)))
        q = q.double().cpu()
        i = 0
        for r, a, b in parts:
            qs[r].append(q[i:i + b - a])
            i += b - a
            at[r] = b
    assert int(err.item()) == 0 and at == list(lens)
    free = [s for s in range(R + 1) if s not in slots]
    assert all((state[s] == 3.0).all() for s in free), "a slot of no request was written"
    got, want = [], []
    for r, n in enumerate(lens):
        t, o = tables[r], [p % ps for p in range(n)]
        idx = [t[p // ps] for p in range(n)]
        got.append((torch.cat(qs[r]), kc[idx, :, o].double().cpu(), vc[idx, :, o].double().cpu()))
        y = plain.causal_conv(rows[r].double(), taps.double())
        v = y[:, (H + G) * d:].reshape(n, G, dv)
        want.append((y[:, :H * d].reshape(n, H, d), y[:, H * d:(H + G) * d].reshape(n, G, d),
                     v if value_eps is None else plain.unit_rms(v, value_eps)))
        if K > 1:       # what the next step would start from
            last = torch.cat([torch.zeros(K - 1, C, dtype=dtype), rows[r]])[-(K - 1):]
            assert torch.equal(state[slots[r]].cpu(), last)
    return got, want


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,K", [(3, 1, 10, 14, 3), (4, 2, 32, 32, 4), (2, 2, 48, 16, 1), (6, 1, 64, 32, 6), (5, 5, 7, 3, 2),
                                        (1, 1, 16, 200, 16), (32, 8, 16, 24, 4)])
def test_convolved_projections_however_the_tokens_are_cut(H, G, d, dv, K, dtype):
    lens = [23, 9, 40]
    whole = [[(0, 23), (1, 9), (2, 40)]]
    cut = [[(0, 2), (2, 1)], [(1, 1), (0, 3), (2, 5)], [(2, 1), (1, 1), (0, 1)], [(0, 17), (1, 7)], [(2, 2)], [(2, 31)]]
    singles = [[(2, 8), (0, 14)]] + [[(2, 1), (1, 1), (0, 1)]] * 9 + [[(2, 1)]] * 23
    for cuts in (whole, cut, singles):
        got, want = _prepare_steps(H, G, d, dv, K, lens, cuts, dtype, seed=H + d)
        for g, w in zip(got, want):
            for a, b in zip(g, w):
                assert (a - b).abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2) * (1 + b.abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dv,K", [(4, 2, 16, 16, 4), (3, 1, 200, 132, 3), (2, 2, 64, 180, 6), (5, 1, 96, 32, 1), (2, 1, 128, 128, 2),
                                        (1, 1, 32, 260, 4), (2, 1, 16, 16, 9)])
@pytest.mark.parametrize("value_eps", [None, 1e-5])
def test_convolution_over_steps_of_many_tokens(H, G, d, dv, K, value_eps, dtype):
    """Warps then take runs of tokens that cross from one request into the next and start in the middle of one; a request
    goes on from a step of single tokens and from a portion shorter than the taps."""
    lens = [700, 3, 1, 130]
    for cuts in ([[(0, 700), (1, 3), (2, 1), (3, 130)]],
                 [[(0, 2), (3, 1)], [(0, 90), (1, 1), (3, 2)], [(0, 1), (3, 1)], [(0, 607), (1, 2), (2, 1), (3, 126)]]):
        got, want = _prepare_steps(H, G, d, dv, K, lens, cuts, dtype, 7, value_eps=value_eps)
        for g, w in zip(got, want):
            assert all((a - b).abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2) * (1 + b.abs().max()) for a, b in zip(g, w))


def test_both_forms_of_the_convolution_give_the_same_bits():
    """Steps of more than 64 tokens take the form in runs, shorter ones a block per token."""
    for dtype in (torch.float32, torch.bfloat16):
        a, _ = _prepare_steps(4, 2, 32, 48, 4, [130], [[(0, 130)]], dtype, 11)
        b, _ = _prepare_steps(4, 2, 32, 48, 4, [130], [[(0, 60)], [(0, 60)], [(0, 10)]], dtype, 11)
        assert all(torch.equal(x, y) for x, y in zip(a[0], b[0]))


def test_a_convolution_takes_no_biases():
    k = _k()
    z = torch.zeros(1, 3 * 16, device=DEV)
    with pytest.raises(k.KernelError):
        k.qkv_prepare(torch.zeros(1, 1, 16, device=DEV), torch.zeros(1, 1, 8, 16, device=DEV), torch.zeros(1, 1, 8, 16, device=DEV), z, None,
                      None, None, _i32([0]), _i32([0]), _i32([[0]]), 1, 1, 1, 16, 16, 0, False, 0, 1e-6, True, _err(),
                      bias=torch.zeros(48, device=DEV), conv=(torch.zeros(1, 48, device=DEV), None, _i32([0, 1]), _i32([0]), True))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [3, 90])
@pytest.mark.parametrize("H,G,d,dv,dims", [(4, 2, 14, 9, 6), (2, 1, 32, 32, 32), (3, 3, 16, 48, 4), (6, 2, 80, 80, 20)])
def test_biases_and_rotation_of_halves(dtype, T, H, G, d, dv, dims):
    base, ps = 300.0, 16
    C = (H + G) * d + G * dv
    x, bias = _rand(T, C, seed=d).to(dtype), _rand(C, seed=1).float()
    pos = torch.arange(1000, 1000 + T)
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    pages = (1000 + T + ps - 1) // ps
    q = torch.full((T, H, d), float("nan"), dtype=dtype, device=DEV)
    kc = torch.full((pages, G, ps, d), float("nan"), dtype=dtype, device=DEV)
    vc = torch.full((pages, G, ps, dv), float("nan"), dtype=dtype, device=DEV)
    err = _err()
    _k().qkv_prepare(q, kc, vc, x.to(DEV), None, None, f.float().to(DEV), pos.int().to(DEV), _i32([0] * T), _i32([list(range(pages))]), pages,
                     H, G, d, dv, dims, False, 0, 1e-6, True, err, bias=bias.to(DEV))
    y = x.double() + bias.double()
    # (the angle is position * frequency in float32; the oracle turns by float64 angles)
    turn = lambda t: plain.rotate_halves(t, pos, dims, base)
    want = (turn(y[:, :H * d].reshape(T, H, d)), turn(y[:, H * d:(H + G) * d].reshape(T, G, d)), y[:, (H + G) * d:].reshape(T, G, dv))
    idx, o = [int(p) // ps for p in pos], [int(p) % ps for p in pos]
    got = (q.double().cpu(), kc[idx, :, o].double().cpu(), vc[idx, :, o].double().cpu())
    assert int(err.item()) == 0
    for a, b in zip(got, want):
        assert (a - b).abs().max() <= (3e-4 if dtype == torch.float32 else 2e-2) * (1 + b.abs().max())


# ---------------------------------------------------------------------------------------------
# attention: a window that keeps the first tokens, a sink, values of another size, outputs that lie apart
# ---------------------------------------------------------------------------------------------
class _Ctx:
    """The fields of a step context that the attention reads, for requests whose keys and values already lie in pages
    (in a scrambled order; pages a windowed cache would have given back are not there) and whose last ``len - start``
    tokens are this step's queries."""

    def __init__(self, ks, vs, starts, ps, dtype, seed, window=None, keep=0):
        from xinfer_b200.parts import LayerCache, Workspace
        lens = [k.shape[0] for k in ks]
        need = [(n + ps - 1) // ps for n in lens]
        total = sum(need) + 3
        order = torch.randperm(total, generator=torch.Generator().manual_seed(seed)).tolist()
        G, d, dv = ks[0].shape[1], ks[0].shape[2], vs[0].shape[2]
        kp = torch.full((total, G, ps, d), float("nan"), dtype=dtype)
        vp = torch.full((total, G, ps, dv), float("nan"), dtype=dtype)
        self.stride = max(need) + 2
        table = torch.full((len(ks), self.stride), -1, dtype=torch.int32)
        at = 0
        for b, (k, v) in enumerate(zip(ks, vs)):
            first = max(0, starts[b] - window + 1) if window else 0        # the first key a query of this step's can see
            for p in range(need[b]):
                if (p + 1) * ps <= first and p * ps >= keep:
                    continue
                table[b, p] = order[at]
                n = min(ps, lens[b] - p * ps)
                kp[order[at], :, :n] = k[p * ps:p * ps + n].transpose(0, 1).to(dtype)
                vp[order[at], :, :n] = v[p * ps:p * ps + n].transpose(0, 1).to(dtype)
                at += 1
        counts = [n - s for n, s in zip(lens, starts)]
        self.bounds = np.concatenate([[0], np.cumsum(counts)]).astype(np.int32)
        self.cache = LayerCache({"k": kp.to(DEV), "v": vp.to(DEV)}, 0, ps)
        self.table = table.to(DEV)
        self.q_start, self.start_pos = _i32(self.bounds.tolist()), _i32(list(starts))
        self.h_q_start, self.h_start_pos = self.bounds, np.asarray(starts, dtype=np.int32)
        self.num_entries = self.real_entries = len(ks)
        self.num_tokens = int(self.bounds[-1])
        self.positions = _i32([s + i for s, c in zip(starts, counts) for i in range(c)])
        self.req_of_token = _i32([b for b, c in enumerate(counts) for _ in range(c)])
        self.fixed_shapes = False
        self.max_context = max(lens)
        self.scratch = {}
        self.workspace = Workspace(DEV)
        self.err = _err()


def _attend(qs, ks, vs, starts, scale, ps, dtype, window=None, keep=0, sink=None, tiled=True, seed=0, out_scale=1.0, apart=0):
    from xinfer_b200.parts import attention_backend as ab
    k = _k()
    ctx = _Ctx(ks, vs, starts, ps, dtype, seed, window, keep)
    q = torch.cat([q[s:] for q, s in zip(qs, starts)]).to(dtype).to(DEV).contiguous()
    T, H, d = q.shape
    dv = vs[0].shape[2]
    wide = torch.full((T, H * dv + apart), 5.0, dtype=dtype, device=DEV)
    out = wide[:, :H * dv].unflatten(1, (H, dv))
    s = sink.float().to(DEV) if sink is not None else None
    G = ks[0].shape[1]
    if tiled:
        assert ab.takes_changed_scores(dtype, H, G, d, ps, dv)
        before = dict(k.launch_counts())
        ab.prepare_step(ctx, dtype, H, G, d, ps, k.mask_code(window), ctx.stride, keep_first=keep, dv=dv)
        ab.attend(out, q, ctx.cache, ctx, ctx.table, ctx.stride, window, scale, sink=s, keep_first=keep, out_scale=out_scale)
        ran = {n for n, c in k.launch_counts().items() if c > before.get(n, 0)}
        assert "attention_plain" not in ran and ran & {"attn_prefill_tc", "attn_decode_tc"}
    else:
        k.attention_plain(out, q, ctx.cache["k"], ctx.cache["v"], ctx.positions, ctx.req_of_token, ctx.table, ctx.stride, window, scale,
                          ctx.err, sink=s, keep_first=keep, out_scale=out_scale)
    torch.cuda.synchronize()
    assert int(ctx.err.item()) == 0
    if apart:
        assert (wide[:, H * dv:] == 5.0).all(), "columns beside the output were written"
    res = out.double().cpu()
    return [res[a:b] for a, b in zip(ctx.bounds[:-1], ctx.bounds[1:])]


def _attend_plain(q, k, v, scale, window, keep, sink):
    return plain.softmax_heads(q, k, v, plain.visible(q.shape[0], window, keep), scale, sink)


FORMS = [(torch.float32, False), (torch.bfloat16, True), (torch.bfloat16, False)]


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("H,G,d,dv,ps", [(4, 2, 32, 32, 8), (6, 2, 96, 96, 16), (3, 1, 16, 80, 32), (8, 1, 128, 64, 16), (5, 5, 48, 112, 64),
                                         (2, 1, 64, 64, 128), (16, 1, 112, 128, 16)])
@pytest.mark.parametrize("window,keep", [(None, 0), (50, 20), (130, 70), (1, 3), (64, 64), (33, 300)])
def test_attention_of_unequal_entries_equals_plain(dtype, tiled, H, G, d, dv, ps, window, keep):
    """Prompt portions of several lengths, one that continues a cached prefix, single tokens and a portion of a few
    tokens, all in one batch, with a sink, a scale and rows that lie apart."""
    lens, starts = [150, 61, 300, 97, 1, 243], [0, 40, 299, 96, 0, 240]
    ks = [_rand(n, G, d, seed=10 * b).to(dtype).double() for b, n in enumerate(lens)]
    vs = [_rand(n, G, dv, seed=10 * b + 2).to(dtype).double() for b, n in enumerate(lens)]
    qs = [(_rand(n, H, d, seed=10 * b + 1) * 1.5).to(dtype).double() for b, n in enumerate(lens)]
    sink = _rand(H, seed=5, scale=2.0).float().double()
    got = _attend(qs, ks, vs, starts, d ** -0.5, ps, dtype, window, keep, sink, tiled, seed=3, out_scale=-0.75, apart=8)
    for q, k, v, s, o in zip(qs, ks, vs, starts, got):
        ref = -0.75 * _attend_plain(q, k, v, d ** -0.5, window, keep, sink)[s:]
        assert (o - ref).abs().max() <= _tol(dtype) * (1 + ref.abs().max())


@pytest.mark.parametrize("tiled", [True, False])
@pytest.mark.parametrize("batch", [1, 8])
def test_single_tokens_over_long_contexts_are_cut_into_pieces_that_agree(tiled, batch):
    """Contexts of thousands of keys are cut into pieces that several blocks take and one merges: the sink counts once, and
    the first tokens and the window are found by whichever piece holds them."""
    H, G, d, dv, ps, window, keep = 4, 2, 64, 64, 16, 3000, 100
    lens = [5000 + 311 * b for b in range(batch)]
    dtype = torch.bfloat16
    ks = [_rand(n, G, d, seed=b).to(dtype).double() for b, n in enumerate(lens)]
    vs = [_rand(n, G, dv, seed=b + 20).to(dtype).double() for b, n in enumerate(lens)]
    qs = [torch.zeros(n, H, d, dtype=F64) for n in lens]
    for b, n in enumerate(lens):
        qs[b][-1] = _rand(H, d, seed=b + 40).to(dtype).double()
        qs[b][-1, 0] = (ks[b][n - 2900, 0] * 2.0).to(dtype).double()      # one key deep in the window
        qs[b][-1, H - 1] = (ks[b][keep - 1, G - 1] * 2.0).to(dtype).double()    # the last kept key
    sink = torch.tensor([0.0, 4.0, 2.0, 30.0], dtype=F64)
    got = _attend(qs, ks, vs, [n - 1 for n in lens], d ** -0.5, ps, dtype, window, keep, sink, tiled, seed=9)
    for q, k, v, n, o in zip(qs, ks, vs, lens, got):
        m = plain.visible(n, window, keep)[-1]
        for h in range(H):
            s = (k[m, h // 2] @ q[-1, h]) * d ** -0.5
            p = torch.softmax(torch.cat([s, sink[h:h + 1]]), 0)[:-1]
            ref = p @ v[m, h // 2]
            assert (o[0, h] - ref).abs().max() <= 3e-2 * (1 + ref.abs().max()), h


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("window,keep", [(48, 16), (64, 64), (2, 65), (200, 1), (11, 40), (130, 0), (70, 128)])
def test_edges_of_the_window_and_of_the_kept_tokens(dtype, tiled, decode, window, keep):
    """One key is made to stand out for the last query: among the kept tokens or inside the window it decides the output,
    one token further it must not be seen."""
    H, G, d, ps, n = 4, 2, 32, 16, 330
    for j, inside in [(n - window, True), (n - window - 1, False), (n - 1, True), (keep - 1, True), (keep, False), (0, keep > 0)]:
        if j < 0 or (j >= keep and n - 1 - j < window) != inside and not (inside and j < keep):
            continue
        k, v = _rand(n, G, d, seed=6).to(dtype).double(), _rand(n, G, d, seed=8).to(dtype).double()
        k[j] = k[j] * 2.0
        q = _rand(n, H, d, seed=7).to(dtype).double()
        q[-1, 0], q[-1, H - 1] = k[j, 0] * 2.0, k[j, G - 1] * 2.0
        start = n - 1 if decode else n - 9
        sink = torch.full((H,), 3.0, dtype=F64)
        got = _attend([q], [k], [v], [start], 1.0, ps, dtype, window, keep, sink, tiled)[0]
        ref = _attend_plain(q, k, v, 1.0, window, keep, sink)[start:]
        assert (got - ref).abs().max() <= _tol(dtype) * (1 + ref.abs().max())
        for h in (0, H - 1):
            carried = (got[-1, h] - v[j, h // 2]).abs().max() < 8e-2 * (1 + v.abs().max())
            assert bool(carried) == inside, (j, inside, h)


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("where", ["first", "second", "page_end", "page_start", "tile_end", "tile_start", "far", "previous"])
def test_one_planted_key_decides_the_output(dtype, tiled, where, decode):
    H, G, d, dv, ps, n = 8, 4, 64, 32, 16, 600
    j = {"first": 0, "second": 1, "page_end": 31, "page_start": 32, "tile_end": 63, "tile_start": 64, "far": n - 517,
         "previous": n - 2}[where]
    k, v = _rand(n, G, d, seed=99).to(dtype).double(), _rand(n, G, dv, seed=97).to(dtype).double()
    q = _rand(n, H, d, seed=98).to(dtype).double()
    q[-1] = k[j].repeat_interleave(2, dim=0)
    start = n - 1 if decode else n - 37
    got = _attend([q], [k], [v], [start], 0.8, ps, dtype, None, 0, None, tiled)[0]
    ref = _attend_plain(q, k, v, 0.8, None, 0, None)[start:]
    assert (got - ref).abs().max() <= _tol(dtype) * (1 + ref.abs().max())
    assert (got[-1, H - 1] - v[j, G - 1]).abs().max() < 8e-2 * (1 + v.abs().max()), "the planted key must carry the output"


@pytest.mark.parametrize("dtype,tiled", FORMS)
@pytest.mark.parametrize("decode", [False, True], ids=["prompt", "decoded"])
@pytest.mark.parametrize("level", [-200.0, -3.0, 0.0, 3.0, 20.0, 400.0])
def test_a_sink_takes_its_share_and_no_more(dtype, tiled, decode, level):
    """Keys that all score alike: the output is the values' mean times n / (n + e^(sink - score)), also for sinks far above
    and far below every score."""
    H, G, d, ps, n = 2, 1, 16, 8, 150
    k, v = torch.zeros(n, G, d, dtype=F64), _rand(n, G, d, seed=1).to(dtype).double()
    k[:, :, 0] = 2.0
    q = torch.zeros(n, H, d, dtype=F64)
    q[:, :, 0] = 1.0
    sink = torch.tensor([level, level - 1.0], dtype=F64)
    start = n - 1 if decode else n - 40
    got = _attend([q], [k], [v], [start], 0.5, ps, dtype, None, 0, sink, tiled)[0]
    ref = _attend_plain(q, k, v, 0.5, None, 0, sink)[start:]
    assert (got - ref).abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2)
    if level == 400.0:
        assert got.abs().max() < 1e-6


# ---------------------------------------------------------------------------------------------
# the matrix memory
# ---------------------------------------------------------------------------------------------
def _memory_steps(H, d, dv, cap, lens, cuts, seed, gates=None, qkv_of=None, spread=3.0):
    """Runs requests through the scan in steps; checks the states, and returns per request o / div as the kernel and as
    the plain recurrence give them."""
    k = _k()
    W = H * (2 * d + dv)
    qkv = [qkv_of(n) if qkv_of else _rand(n, W, seed=seed + i).float() for i, n in enumerate(lens)]
    zs = [gates(n) if gates else _rand(n, 2 * H, seed=seed + 50 + i, scale=spread).float() for i, n in enumerate(lens)]
    bi, bf = _rand(H, seed=seed + 80).float(), (_rand(H, seed=seed + 81) + (0.0 if gates else 2.0)).float()
    if gates:
        bi.zero_(), bf.zero_()
    R = len(lens)
    slots = [R - i for i in range(R)]
    st = {"S": torch.full((R + 1, H, d, dv), 7.0, device=DEV), "n": torch.full((R + 1, H, d), 7.0, device=DEV),
          "m": torch.full((R + 1, H, 2, 2), 7.0, device=DEV)}
    for s in slots:
        for t in st.values():
            t[s].zero_()
    at, outs = [0] * R, [[] for _ in lens]
    gap = 3                                              # columns between v and the gates
    for step in cuts:
        rows = [(r, at[r], at[r] + n) for r, n in step]
        T = sum(n for _, n in step)
        q_start = np.concatenate([[0], np.cumsum([n for _, n in step])]).tolist()
        proj = torch.full((T, W + gap + 2 * H + 1), float("nan"), device=DEV)
        proj[:, :W] = torch.cat([qkv[r][a:b] for r, a, b in rows]).to(DEV)
        proj[:, W + gap:W + gap + 2 * H] = torch.cat([zs[r][a:b] for r, a, b in rows]).to(DEV)
        o = torch.full((T, H * dv), float("nan"), device=DEV)
        div = torch.full((T, H), float("nan"), device=DEV)
        k.matrix_memory(o, div, proj, W + gap, bi.to(DEV), bf.to(DEV), cap, st, _i32(q_start), _i32([a for _, a, _ in rows]),
                        _i32([slots[r] for r, _ in step]), len(step), H, d, dv, d ** -0.5, plain.MEMORY_EPS)
        res = (o.view(T, H, dv) / div[:, :, None]).double().cpu()
        i = 0
        for r, a, b in rows:
            outs[r].append(res[i:i + b - a])
            i += b - a
            at[r] = b
    assert at == list(lens)
    want = []
    for r, (x, z, n) in enumerate(zip(qkv, zs, lens)):
        q, kk, v = x.double().split([H * d, H * d, H * dv], dim=1)
        gi, gf = plain.memory_gates(z[:, :H].double() + bi.double(), z[:, H:].double() + bf.double(), cap)
        o, (S, nn, m) = plain.memory_recurrence(q.reshape(n, H, d) * d ** -0.5, kk.reshape(n, H, d), v.reshape(n, H, dv), gi, gf)
        want.append(o)
        s = slots[r]
        place = st["m"][s].double().cpu()                # two places: the one that stands behind all tokens counts
        held = torch.where(place[:, 0, 0] == n, place[:, 0, 1], place[:, 1, 1])
        assert ((place[:, :, 0] == n).any(dim=1)).all() and (held - m).abs().max() <= 1e-4 * (1 + m.abs().max())
        assert (st["S"][s].double().cpu() - S).abs().max() <= 5e-5 * (1 + S.abs().max())
        assert (st["n"][s].double().cpu() - nn).abs().max() <= 5e-5 * (1 + nn.abs().max())
    free = [s for s in range(R + 1) if s not in slots]
    assert all((t[s] == 7.0).all() for s in free for t in st.values()), "a slot of no request was written"
    return [torch.cat(o) for o in outs], want


@pytest.mark.parametrize("H,d,dv,cap", [(3, 10, 14, 4.0), (1, 7, 5, 15.0), (2, 48, 40, 12.0), (4, 32, 16, 1.0), (1, 16, 300, 9.0),
                                        (2, 130, 64, 30.0), (1, 300, 20, 6.0), (8, 64, 128, 15.0), (2, 1, 1, 2.0), (6, 24, 72, 11.0)])
def test_memory_however_the_tokens_are_cut(H, d, dv, cap):
    lens = [70, 33, 5]
    for cuts in ([[(0, 70), (1, 33), (2, 5)]],
                 [[(0, 2), (1, 17)], [(2, 3), (0, 31)], [(0, 1), (1, 1), (2, 1)], [(1, 15), (0, 36), (2, 1)]],
                 [[(0, 60), (1, 30)]] + [[(0, 1), (2, 1)]] * 5 + [[(0, 1), (1, 1)]] * 3 + [[(0, 1)]] * 2):
        got, want = _memory_steps(H, d, dv, cap, lens, cuts, seed=H + d)
        for g, w in zip(got, want):
            assert (g - w).abs().max() <= 1e-4 * (1 + w.abs().max())


def test_a_token_written_long_ago_is_read_while_its_gates_let_it():
    """One token writes with a strong input gate a key that nothing else uses; forget gates of one keep it for hundreds of
    tokens (and many tiles); a head whose forget gates are weak has lost it."""
    H, d, dv, n = 2, 12, 8, 500

    def qkv(T):
        x = torch.zeros(T, H * (2 * d + dv))
        q, k, v = x[:, :H * d].view(T, H, d), x[:, H * d:2 * H * d].view(T, H, d), x[:, 2 * H * d:].view(T, H, dv)
        q[:, :, 1:] = _rand(T, H, d - 1, seed=4).float()
        k[:, :, 1:] = _rand(T, H, d - 1, seed=5).float()
        v[:] = _rand(T, H, dv, seed=6).float()
        k[3] = 0
        k[3, :, 0] = 1.0
        q[n - 1] = 0
        q[n - 1, :, 0] = d ** 0.5
        return x

    def gates(T):
        z = torch.full((T, 2 * H), -9.0)
        z[3, :H] = 9.0
        z[:, H] = 60.0                                   # head 0 keeps nearly all
        z[:, H + 1] = -1.0                               # head 1 forgets
        return z

    for cuts in ([[(0, n)]], [[(0, 5)], [(0, n - 12)]] + [[(0, 1)]] * 7):
        got, want = _memory_steps(H, d, dv, 20.0, [n], cuts, seed=0, gates=gates, qkv_of=qkv)
        v3 = qkv(n)[3, 2 * H * d:].view(H, dv).double()
        assert (got[0][n - 1, 0] - v3[0]).abs().max() < 1e-3 and got[0][n - 1, 1].abs().max() < 1e-2
        assert (got[0] - want[0]).abs().max() <= 1e-4 * (1 + want[0].abs().max())


@pytest.mark.parametrize("z_i,z_f", [(80.0, 80.0), (-80.0, -80.0), (80.0, -80.0), (-80.0, 80.0)])
def test_memory_gates_far_out_stay_in_range(z_i, z_f):
    """Pre-activations far beyond the cap: nothing overflows, also over hundreds of tokens."""
    H, d, dv, n, cap = 2, 16, 8, 300, 25.0

    def gates(T):
        return torch.cat([torch.full((T, H), z_i), torch.full((T, H), z_f)], dim=1)

    got, want = _memory_steps(H, d, dv, cap, [n], [[(0, 100)], [(0, 1)], [(0, n - 101)]], seed=3, gates=gates)
    assert torch.isfinite(got[0]).all() and (got[0] - want[0]).abs().max() <= 1e-4 * (1 + want[0].abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dv", [(3, 14), (2, 64), (1, 200), (1, 700)])
def test_division_norm_per_head_and_gate_into_a_column_range(dtype, H, dv):
    T, eps = 11, 1e-5
    o, row = _rand(T, H * dv, seed=1).float(), _rand(T, H * dv + 7, seed=2, scale=2.0).float()
    w, div = (1 + _rand(H * dv, seed=3, scale=0.3)).float(), _rand(T, H, seed=4).abs().float() + 0.1
    div[3] = 1e4                                         # a head whose norm's eps decides
    wide = torch.full((T, H * dv + 6), 5.0, dtype=dtype, device=DEV)
    _k().gated_head_norm(wide[:, 4:4 + H * dv], o.to(DEV), row.to(DEV), 7, w.to(DEV), dv, eps, gate_after=True, div=div.to(DEV),
                         out_scale=-1.5)
    g = row.double()[:, 7:]
    x = plain.unit_rms(o.double().view(T, H, dv) / div.double()[:, :, None], eps).reshape(T, H * dv)
    want = -1.5 * x * w.double() * torch.sigmoid(g)
    got = wide.double().cpu()
    assert (got[:, :4] == 5.0).all() and (got[:, 4 + H * dv:] == 5.0).all()
    assert (got[:, 4:4 + H * dv] - want).abs().max() <= (1e-5 if dtype == torch.float32 else 1e-2) * (1 + want.abs().max())


# ---------------------------------------------------------------------------------------------
# the router with groups and the experts
# ---------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("E,top,groups,keep", [(6, 2, 3, 2), (12, 4, 4, 3), (1, 1, 1, 1), (8, 1, 2, 1), (16, 4, 8, 2), (9, 2, 3, 1), (7, 7, 1, 1)])
def test_softmax_router_among_groups_chooses_as_plain(dtype, E, top, groups, keep):
    T, K = 61, 52
    h, w = _rand(T, K, seed=E).to(dtype), _rand(E, K, seed=E + 1, scale=0.4).float()
    choice = torch.full((T, top), -7, dtype=torch.int32, device=DEV)
    weight = torch.full((T, top), float("nan"), dtype=torch.float32, device=DEV)
    req = torch.zeros(T, dtype=torch.int32)
    req[5] = -1                                          # a padding token takes part in nothing
    _k().expert_router(choice, weight, h.to(DEV), w.to(DEV), None, req.to(DEV), top, groups, keep, 1, renormalize=True, softmax=True,
                       renormalize_eps=1e-20)
    idx, wt = plain.route(h.double(), w.double(), dict(experts=E, top=top, groups=dict(count=groups, keep=keep)))
    got_i, got_w = choice.cpu(), weight.double().cpu()
    for t in range(T):
        if t == 5:
            assert got_w[t].abs().max() == 0
            continue
        assert got_i[t].tolist() == idx[t].tolist(), t
        assert (got_w[t] - wt[t]).abs().max() < 2e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [1, 3, 70])
@pytest.mark.parametrize("E,top,groups,keep,limit", [(6, 2, 3, 2, 0.8), (1, 1, 1, 1, 2.0), (8, 4, 2, 1, 0.3), (4, 3, 1, 1, 7.0)])
def test_routed_experts_part_equals_plain(dtype, T, E, top, groups, keep, limit):
    from xinfer_b200.config.plan import RoutedExpertsSpec
    from xinfer_b200.parts import Workspace, build_part
    from xinfer_b200.parts.base import StepContext
    W, Fi = 48, 24
    mlp = dict(kind="moe", expert=dict(ff=Fi, limit=limit), router=dict(experts=E, top=top, groups=dict(count=groups, keep=keep)))
    w = {}
    for i, n in enumerate(f"m.e{e}.{n}" for e in range(E) for n in ("gate", "up", "down")):
        w[n] = _rand(*((W, Fi) if n.endswith("down") else (Fi, W)), seed=100 + i, scale=0.2).to(dtype).double()
    w["m.router"] = _rand(E, W, seed=7, scale=0.3).to(dtype).double()

    class Store:
        def get(self, name, device, dt, operand=False, columns=None):
            return w[name].to(dt).to(device)

    spec = RoutedExpertsSpec(kind="routed_experts", hidden=W, intermediate=Fi, experts=E, top=top, groups=groups, keep=keep, group_best=1,
                             correction=False, renormalize=True, score="softmax", renormalize_eps=1e-20, activation="swish_clamp",
                             act_params=(limit, plain.SWISH_ALPHA))
    part = build_part("feed_forward", spec, "m.", dtype, DEV)
    part.load(Store())
    x = _rand(T, W, seed=T).to(dtype)
    req = torch.zeros(T, dtype=torch.int32)
    if T > 1:
        req[1] = -1
    ctx = StepContext(dtype=dtype, device=torch.device(DEV), num_tokens=T, num_entries=1, token_ids=_i32([0] * T),
                      positions=_i32(list(range(T))), req_of_token=req.to(DEV), q_start=_i32([0, T]), start_pos=_i32([0]),
                      slots=_i32([0]), logit_rows=_i32([0]), num_logit_rows=0, tables=[], strides=[], err=_err(),
                      workspace=Workspace(DEV), branch_dtype=torch.float32)
    want = plain.routed_experts(x.double(), w, "m.", mlp)
    keep_rows = [t for t in range(T) if t != 1]
    out = part.forward(x.to(DEV), ctx).double().cpu()
    assert int(ctx.err.item()) == 0
    assert (out[keep_rows] - want[keep_rows]).abs().max() <= (2e-5 if dtype == torch.float32 else 4e-2) * (1 + want.abs().max())


# ---------------------------------------------------------------------------------------------
# whole models: every way of cutting, pages and slots used again, layer by layer, generation
# ---------------------------------------------------------------------------------------------
LENGTHS = {"A": [70, 45, 130, 33], "B": [97, 41, 260, 150], "C": [170, 1, 75, 58], "D": [90, 2, 51, 140], "E": [40, 21, 70], "F": [60, 31, 85]}


def _tolerance(dtype, ref, cfg=None, w=None, p=None, routes=None):
    """float32: a small share of the logits' spread (the engine's float32 against float64).  bfloat16: three times what
    rounding alone causes - the largest row error of the plain run that rounds activations to bfloat16 where an engine
    stores them (along the same experts: another choice is no rounding error)."""
    spread = max(float(np.std(ref)), 1e-3)
    if dtype == "float32":
        return 1e-4 * spread
    rounded = plain.forward(cfg, w, p, round_to=torch.bfloat16, routes=routes, slack=float("inf")).numpy()
    return max(3.0 * max(row_error(rounded[i], ref[i]) for i in range(len(p))), 1e-3 * spread)


def _store(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


@pytest.mark.parametrize("name", sorted(TINY_D))
def test_every_way_of_cutting_gives_the_plain_logits_in_float32_through_the_replay_program(name, tmp_path):
    dtype = "float32"
    folder = make_folder(str(tmp_path / "model"), name, _store(dtype))
    ps = prompts(name, LENGTHS[name])
    tb = build_all_modes(ps, seed=len(name))
    out = run_trace(folder, dtype, tb.steps, str(tmp_path / "out"), max_tokens=tb.peak, page_size=TINY_D[name][2], max_num_seqs=4)
    cfg, w = plain.load_folder(folder)
    ref = [plain.forward(cfg, w, p).numpy() for p in ps]
    tol = [_tolerance(dtype, r) for r in ref]
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
    activations may decide a router's close call the other way, after which the request is another computation: the
    engine's choices are recorded, checked to differ from the plain ones by close calls only, and followed by the plain
    run (in float32 nothing is close: the slack is a rounding error's)."""
    L = len(cfg["layers"])
    moe_runs = [i for i in range(L) if cfg["layers"][i].get("mlp") is not None]
    out, routes = replay_with_routes(runner, tb.steps, moe_runs)
    slack = 1e-4 if dtype == "float32" else 0.5          # (a router's logits are a few units apart)
    ref, tol = {}, {}         # per request id of the trace: the plain logits along the engine's routes

    def plain_of(rid, i):
        if rid not in ref:
            given = [routes[rid].get(run) for run in range(L)]
            ref[rid] = None
            x = _plain_along(cfg, w, ps[i], given, slack)
            ref[rid] = x
            tol[rid] = _tolerance(dtype, x, cfg, w, ps[i], given)
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


_runs = {}


def _plain_along(cfg, w, p, given, slack):
    """The plain logits along an engine's routes; runs of the same prompt with the same choices are made once."""
    key = (id(w), tuple(p), tuple(None if g is None else tuple(map(tuple, g.sort(dim=1).values.tolist())) for g in given))
    if key not in _runs:
        if len(_runs) > 64:
            _runs.clear()
        _runs[key] = (w, plain.forward(cfg, w, p, routes=given, slack=slack).numpy())
    return _runs[key][1]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(TINY_D))
def test_every_way_of_cutting_gives_the_plain_logits(name, dtype, tmp_path):
    """Every request whole, with its tail token by token, in portions, and four at a time over a pool of the live
    requests' size, against the plain run."""
    from xinfer_b200.engine.runner import ModelRunner
    folder = make_folder(str(tmp_path / "model"), name, _store(dtype))
    ps = prompts(name, LENGTHS[name])
    tb = build_all_modes(ps, seed=len(name))
    page = TINY_D[name][2]
    runner = ModelRunner(folder, dtype, block_size=page, num_blocks=(tb.peak + page - 1) // page, max_num_seqs=4)
    cfg, w = plain.load_folder(folder)
    worst = _check_trace(name, dtype, runner, tb, ps, cfg, w)
    print(name, dtype, "worst error / tolerance per mode:", {k: f"{v:.3g}" for k, v in worst.items()})


@pytest.mark.parametrize("name,dtype", [("A", "float32"), ("B", "bfloat16"), ("C", "bfloat16"), ("D", "float32")])
def test_freed_pages_and_slots_are_used_again_and_nothing_stale_is_read(name, dtype, tmp_path):
    """Pages that go back to the pool are filled with NaN before the next step (also the pages between the kept tokens and
    the window, which go back while a request runs), and every state row starts out as junk.  Requests pass through four
    slots and a pool of the live requests' size: the logits stay the plain ones and stay finite."""
    from xinfer_b200.engine.runner import ModelRunner
    folder = make_folder(str(tmp_path / "model"), name, _store(dtype))
    ps = prompts(name, LENGTHS[name])
    tb = build_all_modes(ps, seed=3)
    page = TINY_D[name][2]
    runner = ModelRunner(folder, dtype, block_size=page, num_blocks=(tb.peak + page - 1) // page, max_num_seqs=4,
                         poison_freed_pages=True)
    for t in runner.state.tables.values():
        t.fill_(1e4)
    cfg, w = plain.load_folder(folder)
    _check_trace(name, dtype, runner, tb, ps, cfg, w)
    assert runner.pages_poisoned > runner.num_blocks


@pytest.mark.parametrize("name", sorted(TINY_D))
def test_layers_one_by_one_in_float32(name, tmp_path):
    """The sum of the residual streams after every layer against the plain one, a prompt in two portions."""
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
        rec.append(out.x.double().sum(dim=1).cpu())
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
        assert got.dtype == F64 and (got - ref).abs().max() <= 5e-5 * (1 + ref.abs().max()), f"layer {i}"


def test_the_streams_are_float32_and_the_fused_and_fast_kernels_run_in_bfloat16(tmp_path):
    from xinfer_b200 import kernels
    from xinfer_b200.engine.runner import ModelRunner, StepInput
    folder = make_folder(str(tmp_path / "model"), "B", torch.bfloat16)
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
    # six layers (two without experts): ten halves and the final norm, one kernel each for all stream arithmetic
    for used in (first, then):
        assert used["stream_mix"] == 11 and not set(used) & {"add_f32", "rmsnorm_f32", "rms_chain", "attention_plain", "attn_talking_mma"}
        assert used["qkv_prepare"] == 6 and used["matrix_memory"] == 3 and used["gated_head_norm"] == 3
    assert first["attn_prefill_tc"] == 6 and then["attn_decode_tc"] == 6
    # one token per request: the convolution's inputs are kept in the same launch
    assert first["conv_state"] == 2 and "conv_state" not in then
    assert "expert_gemm_mma" in first and then["expert_select_gate"] == 4


def test_layers_that_share_weights_keep_caches_and_states_of_their_own(tmp_path):
    from xinfer_b200.engine.runner import ModelRunner
    folder = make_folder(str(tmp_path / "model"), "A", torch.bfloat16)
    runner = ModelRunner(folder, "bfloat16", block_size=8, num_blocks=32, max_num_seqs=2)
    caches, states = runner.layer_caches, runner.layer_states
    assert all(c is not None for c in caches) and len({c["k"].data_ptr() for c in caches}) == 6
    assert states[1]["right.S"].data_ptr() != states[3]["right.S"].data_ptr() and states[2] is None
    assert states[0]["conv"].data_ptr() != states[4]["conv"].data_ptr() and states[0]["conv"].dtype == torch.bfloat16
    # runs of one kind share a page pool; the window that keeps first tokens has one of its own
    assert caches[0].group == caches[2].group == caches[4].group != caches[1].group == caches[3].group
    g = runner.cache.groups[caches[1].group]
    assert (g.window, g.keep_first) == (11, 5)
    cfg, w = plain.load_folder(folder)
    assert runner.model.weight_bytes() >= 2 * sum(t.numel() for t in w.values())


def _engine(folder, dtype, page, **kw):
    from xinfer_b200 import Engine, EngineConfig
    opts = dict(weight_path=folder, block_size=page, num_blocks=96, max_num_seqs=4, max_num_batched_tokens=64,
                prefill_chunk_size=16, disable_cuda_graph=True, max_model_len=1024)
    opts.update(kw)
    return Engine(EngineConfig(**opts), dtype)


@pytest.mark.parametrize("name", ["A", "C", "D"])
def test_greedy_generation_in_float32_equals_plain(name, tmp_path):
    from xinfer_b200 import SamplingParams
    folder = make_folder(str(tmp_path / "model"), name, torch.float32)
    cfg, w = plain.load_folder(folder)
    ps = prompts(name, [1, 5, 23, 40, 9, 17])       # six requests over four slots, prompts in portions of 16
    eng = _engine(folder, "f32", TINY_D[name][2])
    outs = eng.generate_sync(SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True), ps)
    for p, o in zip(ps, outs):
        assert o.decode_output == plain.greedy(cfg, w, p, 12)


@pytest.mark.parametrize("graphs", [False, True], ids=["launched", "cuda_graph"])
@pytest.mark.parametrize("name", ["F"])
def test_long_greedy_decoding_in_bfloat16_follows_the_plain_logits(name, graphs, tmp_path):
    """Each generated token is checked against the plain logits of the sequence the engine produced (bfloat16 may flip a
    near-tie): it must be the best token up to the drift.  Long enough for many pages per request and for windows to pass
    over decoded tokens."""
    from xinfer_b200 import SamplingParams
    folder = make_folder(str(tmp_path / "model"), name, torch.bfloat16)
    cfg, w = plain.load_folder(folder)
    ps = prompts(name, [3, 30, 61])
    eng = _engine(folder, "bf16", TINY_D[name][2], disable_cuda_graph=not graphs)
    outs = eng.generate_sync(SamplingParams(max_tokens=150, ignore_eos=True), ps)
    assert eng.runner.last_used_graph == graphs
    for p, o in zip(ps, outs):
        assert o.decoded_length == 150
        seq = p + o.decode_output
        ref = plain.forward(cfg, w, seq)
        slack = 2 * 3.0 * float((plain.forward(cfg, w, seq, round_to=torch.bfloat16) - ref).abs().max())
        assert slack < 0.2 * float(ref.max() - ref.min()), "the drift is too large for this to show anything"
        for i, tok in enumerate(o.decode_output):
            row = ref[len(p) + i - 1]
            assert row[tok] >= row.max() - slack, (i, tok)


def test_a_replayed_decode_step_equals_a_launched_one(tmp_path):
    """A CUDA graph is captured by running the step for real a few times; the memories, the convolutions' inputs and the
    token before go back to what they were."""
    from xinfer_b200 import SamplingParams
    folder = make_folder(str(tmp_path / "model"), "F", torch.bfloat16)
    ps = prompts("F", [7, 33, 18])
    outs = []
    for graphs in (False, True):
        eng = _engine(folder, "bf16", 16, disable_cuda_graph=not graphs)
        outs.append([o.decode_output for o in eng.generate_sync(SamplingParams(max_tokens=40, ignore_eos=True), ps)])
        del eng
    assert outs[0] == outs[1]


def test_command_line_writes_a_random_folder_and_generates_from_it(tmp_path, capsys):
    """The command line end to end: a folder from a configuration and a seed, then generation from given ids (equal to the
    plain continuation in float32) and from a seeded prompt of a given length."""
    import json
    from xinfer_b200.cli import main
    config = tmp_path / "config.json"
    config.write_text(json.dumps(TINY_D["A"][0]))
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
