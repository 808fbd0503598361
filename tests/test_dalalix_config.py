"""The Dalalix configuration reader, its plan and the plain implementation's pieces at hand-computed points (CPU)."""
import copy
import math

import pytest
import torch

import plain_dalalix as plain
from dalalix_models import TINY_D
from xinfer_b200.cache import CacheGroup, CacheManager
from xinfer_b200.config import BlockOp, BlockSpec, ConfigError, NormSpec, config_from_dict
from xinfer_b200.config.dalalix import SWISH_ALPHA, DalalixConfig
from xinfer_b200.config.plan import StreamMixSpec
from xinfer_b200.models.decoder import model_weight_specs
from xinfer_b200.parts.rope import inv_frequencies

F64 = torch.float64


def _plan(cfg):
    entry, c = config_from_dict(cfg)
    assert isinstance(c, DalalixConfig)
    return entry.plan_of(c)


def _check_attention(a, m):
    assert a.kind == "talking_attention" and not a.talking_heads and not a.sink and not a.qk_norm
    assert (a.num_heads, a.num_kv_heads, a.head_dim, a.value_dim, a.scale) == (
        m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"])


@pytest.mark.parametrize("name", sorted(TINY_D))
def test_every_key_reaches_a_spec(name):
    cfg = TINY_D[name][0]
    plan = _plan(cfg)
    assert plan.vocab_size == cfg["vocab"] and plan.hidden == cfg["width"] and plan.head_name == "head"
    assert plan.residual_dtype == "float32" and plan.streams == cfg["streams"] and plan.logit_softcap == cfg.get("logit_softcap")
    assert plan.final_norm.eps == cfg["norm"]["eps"]
    b = (cfg.get("embedding") or {}).get("bigram")
    assert (plan.pair_embedding is None) == (b is None)
    if b:
        p = plan.pair_embedding
        assert (p.buckets, p.mul_prev, p.mul_cur) == (b["buckets"], b["mul_prev"], b["mul_cur"])
    assert len(plan.runs) == len(cfg["layers"])
    for i, (layer, run) in enumerate(zip(cfg["layers"], plan.runs)):
        block, m = plan.blocks[run.block], layer["mixer"]
        assert block.prefix == f"l{layer.get('weights_of', i)}." and run.cache_from is None
        reads = [o for o in block.program if o.op == "norm"]
        writes = [o for o in block.program if o.op == "add"]
        want = ["norm1"] if layer["mlp"] is None else ["norm1", "norm2"]
        assert [o.name for o in reads] == want and len(writes) == len(want)
        for q, (r, w) in enumerate(zip(reads, writes), 1):
            assert r.mix == w.mix == StreamMixSpec(cfg["streams"], (f"hc{q}.in", f"hc{q}.mix", f"hc{q}.out"))
            assert r.src == w.dst == "x" and r.spec.eps == cfg["norm"]["eps"]
        a = block.mixer
        if layer["type"] == "attention":
            _check_attention(a, m)
            assert a.conv == m["conv"] and a.value_norm_eps == cfg["norm"]["eps"] and a.gate_name == "g" and not a.gate_per_head
            assert a.rope is None and a.window is None and a.bias_suffix is None and a.sink_name is None
        elif layer["type"] == "attention_2":
            _check_attention(a, m)
            assert a.bias_suffix == ".b" and not a.out_bias and a.rope is None and a.window is None and a.conv is None
            assert a.value_norm_eps is None and a.gate_name is None and a.sink_name is None
        else:
            l, r = a.left, a.right
            _check_attention(l, m["left"])
            assert (a.left_scale, a.right_scale) == (m["left_scale"], m["right_scale"]) and a.out_norms is None
            assert (l.window, l.keep_first) == (m["left"]["mask"]["size"], m["left"]["mask"]["keep_first"])
            assert l.sink_name == "sink" and l.bias_suffix == ".b" and l.gate_name is None and l.conv is None
            rot = m["left"].get("rot")
            assert (l.rope is None) == (rot is None)
            if rot:
                assert (l.rope.rotary_dim, l.rope.theta, l.rope.layout) == (rot["dims"], rot["base"], "neox")
            assert (r.heads, r.head_dim, r.v_head_dim, r.gate_cap) == tuple(m["right"][k] for k in ("heads", "dim", "vdim", "gate_cap"))
            assert r.eps == cfg["norm"]["eps"] and r.divisor_eps == plain.MEMORY_EPS
        f = block.feed_forward
        if layer["mlp"] is None:
            assert f is None
        else:
            e, r = layer["mlp"]["expert"], layer["mlp"]["router"]
            g = r.get("groups") or dict(count=1, keep=1)
            assert (f.intermediate, f.experts, f.top, f.groups, f.keep, f.group_best) == (e["ff"], r["experts"], r["top"], g["count"], g["keep"], 1)
            assert f.score == "softmax" and f.renormalize and f.renormalize_eps == plain.WEIGHT_SUM_EPS and not f.correction
            assert f.activation == "swish_clamp" and f.act_params == (e["limit"], SWISH_ALPHA) and f.shared is None


def test_layers_that_use_weights_again_share_a_block_and_nothing_else():
    plan = _plan(TINY_D["A"][0])
    assert [r.block for r in plan.runs] == [0, 1, 2, 1, 0, 1] and len(plan.blocks) == 3
    plan = _plan(TINY_D["D"][0])      # also of a later layer
    assert [plan.blocks[r.block].prefix for r in plan.runs] == ["l3.", "l1.", "l2.", "l3.", "l4.", "l2."]


def test_declared_tensors():
    names = {s.name: tuple(s.shape) for s in model_weight_specs(_plan(TINY_D["A"][0]))}
    assert names["embed"] == (83, 48) and names["bigram"] == (38, 48) and names["head"] == (83, 48) and names["final.norm"] == (48,)
    assert not any(n.startswith(("l3.", "l4.", "l5.")) for n in names)
    assert names["l0.mix.q"] == (30, 48) and names["l0.mix.k"] == (10, 48) and names["l0.mix.v"] == (14, 48)
    assert names["l0.mix.q.conv"] == (30, 3) and names["l0.mix.v.conv"] == (14, 3) and names["l0.mix.g"] == (42, 48)
    assert names["l0.mix.o"] == (48, 42) and "l0.mix.q.b" not in names
    assert names["l2.mix.q.b"] == (35,) and names["l2.mix.v.b"] == (60,) and "l2.mix.o.b" not in names and "l2.mix.g" not in names
    assert names["l1.mix.left.sink"] == (4,) and names["l1.mix.left.k.b"] == (28,) and names["l1.mix.left.o"] == (48, 36)
    assert names["l1.mix.right.i"] == (3, 48) and names["l1.mix.right.f.b"] == (3,) and names["l1.mix.right.norm"] == (15,)
    assert names["l1.mix.right.g"] == (15, 48) and names["l1.mix.right.o"] == (48, 15) and names["l1.mix.right.q"] == (21, 48)
    assert names["l0.hc1.in"] == (3,) and names["l0.hc1.mix"] == (3, 3) and names["l0.hc2.out"] == (3,)
    assert not any(n.startswith(("l2.hc2", "l2.norm2", "l2.mlp")) for n in names) and names["l0.mlp.router"] == (6, 48)
    assert names["l1.mlp.e4.down"] == (48, 24)
    assert "bigram" not in {s.name for s in model_weight_specs(_plan(TINY_D["C"][0]))}


def test_named_errors():
    base = TINY_D["A"][0]

    def broken(change):
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(ConfigError) as e:
            config_from_dict(cfg)
        return str(e.value)

    assert "streams" in broken(lambda c: c.pop("streams"))
    assert "norm.eps" in broken(lambda c: c["norm"].update(eps=0))
    assert "embedding.bigram.mul_prev" in broken(lambda c: c["embedding"]["bigram"].pop("mul_prev"))
    assert "layers[0].mixer.conv" in broken(lambda c: c["layers"][0]["mixer"].pop("conv"))
    assert "layers[0].mixer.heads" in broken(lambda c: c["layers"][0]["mixer"].update(heads=4, kv_heads=3))
    assert "layers[2].mixer.scale" in broken(lambda c: c["layers"][2]["mixer"].pop("scale"))
    assert "layers[1].mixer.left.mask.size" in broken(lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0))
    assert "layers[1].mixer.left.mask.keep_first" in broken(lambda c: c["layers"][1]["mixer"]["left"]["mask"].pop("keep_first"))
    assert "layers[1].mixer.left.rot.dims" in broken(lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=16))
    assert "layers[1].mixer.right.gate_cap" in broken(lambda c: c["layers"][1]["mixer"]["right"].update(gate_cap=-1))
    assert "layers[1].mixer.right_scale" in broken(lambda c: c["layers"][1]["mixer"].pop("right_scale"))
    assert "layers[2].type" in broken(lambda c: c["layers"][2].update(type="gla"))
    assert "layers[0].mlp.kind" in broken(lambda c: c["layers"][0]["mlp"].update(kind="dense"))
    assert "layers[0].mlp.expert.limit" in broken(lambda c: c["layers"][0]["mlp"]["expert"].pop("limit"))
    assert "layers[0].mlp.router.top" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=5))     # two groups of two
    assert "layers[0].mlp.router.experts" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(experts=7))
    assert "weights_of" in broken(lambda c: c["layers"][3].update(weights_of=4))        # a layer without its own
    assert "weights_of" in broken(lambda c: c["layers"][3].update(weights_of=9))
    assert "layer 3" in broken(lambda c: c["layers"][3].update(weights_of=0))           # another type


def test_blocks_that_disagree_about_the_streams_are_refused():
    mix, norm = StreamMixSpec(2, ("r", "m", "w")), NormSpec(kind="rmsnorm", dim=8)
    part = NormSpec(kind="swiglu", dim=8)
    ok = (BlockOp("norm", "x", "h", norm, mix=mix), BlockOp("feed_forward", "h", "f", part), BlockOp("add", "f", "x", mix=mix))
    spec = BlockSpec("b.", ok)
    spec.validate()
    assert spec.streams == 2
    for bad in ((ok[0], ok[1], BlockOp("add", "f", "x")), (BlockOp("norm", "x", "h", norm), ok[1], ok[2]),
                (ok[0], ok[1], BlockOp("add", "f", "x", scale=0.5, mix=mix)),
                (ok[0], ok[1], BlockOp("add", "f", "x", mix=StreamMixSpec(3, ("r", "m", "w")))),
                (ok[0], BlockOp("feed_forward", "x", "f", part), ok[2]),
                (ok[0], BlockOp("norm", "h", "g", norm, mix=mix), ok[1], ok[2])):
        with pytest.raises(ValueError):
            BlockSpec("b.", bad).validate()


@pytest.mark.parametrize("dims,base", [(20, 9000.0), (6, 40.0), (128, 1e6), (2, 3.0)])
def test_frequencies_of_the_product_equal_the_plain_ones(dims, base):
    want = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    got = torch.from_numpy(inv_frequencies(base, dims, None, True)).double()
    assert ((got - want).abs() <= 1e-7 * want).all()


@pytest.mark.parametrize("page,window,keep", [(8, 20, 5), (8, 20, 8), (8, 20, 9), (16, 1, 40), (4, 30, 1), (8, 200, 16)])
def test_kept_pages_stay_while_the_window_moves_on(page, window, keep):
    cm = CacheManager([CacheGroup(page, 64, window, keep)], max_requests=2)
    slot, total = cm.open_request(), 300
    n = 0
    while n < total:
        step = min(7, total - n)
        held = len([p for p in cm.table(slot) if p >= 0])
        if not cm.extend(slot, n + step):
            raise AssertionError(f"{held} pages held of 64")
        n += step
        cm.advance(slot, n)
        table = cm.table(slot)
        first = max(0, n - window + 1)          # the first key in the window of the next query
        for i, p in enumerate(table):
            needed = i * page < keep or (i + 1) * page > first
            assert (p >= 0) == needed, (n, i)
        cm.check_consistent()
    cm.close_request(slot)
    assert cm.free_pages(0) == 64


def test_plain_pieces_at_hand_computed_points():
    # the pair table: the hash of (token before, token), the last row first
    assert plain.pair_rows([3, 4, 3], dict(buckets=10, mul_prev=7, mul_cur=2)) == [10, 29 % 10, 34 % 10]
    # streams: M is indexed [from, to], all written at once from the old ones
    X = torch.tensor([[[1.0]], [[10.0]]], dtype=F64)
    M = torch.tensor([[0.0, 2.0], [3.0, 0.0]], dtype=F64)
    Y = plain.write_streams(X, M, torch.tensor([1.0, -1.0], dtype=F64), torch.tensor([[5.0]], dtype=F64))
    assert Y.flatten().tolist() == [35.0, -3.0]
    assert float(plain.read_streams(Y, torch.tensor([1.0, 2.0], dtype=F64))) == 29.0
    # the window counts the token itself; the first tokens stay visible, never those ahead
    m = plain.visible(6, 2, 2)
    assert m[5].tolist() == [True, True, False, False, True, True] and m[0].tolist() == [True] + [False] * 5
    assert plain.visible(3)[2].all() and not plain.visible(3, 2, 0)[2, 0]
    # a sink takes weight and gives no value
    one = torch.ones(1, 1, 1, dtype=F64)
    o = plain.softmax_heads(one, one, one * 8.0, plain.visible(1), math.log(3.0), torch.tensor([0.0], dtype=F64))
    assert abs(float(o) - 6.0) < 1e-12
    # a quarter turn of the pair (0, 2) of four rotated channels
    y = plain.rotate_halves(torch.tensor([[[3.0, 0.0, 4.0, 0.0, 9.0]]], dtype=F64), torch.tensor([math.pi / 2]), 4, 10.0)
    assert (y - torch.tensor([[[-4.0, 0.0, 3.0, 0.0, 9.0]]], dtype=F64)).abs().max() < 1e-6
    # the convolution: zeros before the start, the last tap weighs the token itself
    x = torch.tensor([[1.0], [2.0], [5.0]], dtype=F64)
    assert plain.causal_conv(x, torch.tensor([[10.0, 100.0]], dtype=F64)).flatten().tolist() == [100.0, 210.0, 520.0]


def test_plain_memory_starts_its_maximum_at_zero_and_never_divides_by_less():
    one = lambda v: torch.tensor([[[float(v)]]], dtype=F64)
    g = lambda v: torch.tensor([[float(v)]], dtype=F64)
    # i = -5, f = -1: m' = max(-1, -5) = -1, S = e^(-5 + 1) k v, n = e^-4 k, divisor max(|n q|, e^1)
    o, (S, n, m) = plain.memory_recurrence(one(2), one(3), one(7), g(-5), g(-1))
    assert float(m) == -1.0 and abs(float(n) - 3 * math.exp(-4)) < 1e-15
    assert abs(float(o) - 2 * 21 * math.exp(-4) / (math.exp(1) + 1e-6)) < 1e-12
    # a strong input takes over: i = 4, f = 0 gives m' = 4
    _, (S2, n2, m2) = plain.memory_recurrence(one(1), one(1), one(1), g(4), g(0), (S, n, m))
    assert float(m2) == 4.0 and abs(float(S2) - (math.exp(-5) * float(S) + 1.0)) < 1e-12
    i, f = plain.memory_gates(torch.tensor(1e9, dtype=F64), torch.tensor(0.0, dtype=F64), 3.0)
    assert float(i) == 3.0 and abs(float(f) + math.log(2.0)) < 1e-15
    # the recurrence carried over a cut equals the whole
    gen = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, d, generator=gen, dtype=F64) for d in (3, 3, 4))
    i, f = torch.randn(9, 2, generator=gen, dtype=F64), -torch.rand(9, 2, generator=gen, dtype=F64)
    o, st = plain.memory_recurrence(q, k, v, i, f)
    o1, s1 = plain.memory_recurrence(q[:4], k[:4], v[:4], i[:4], f[:4])
    o2, s2 = plain.memory_recurrence(q[4:], k[4:], v[4:], i[4:], f[4:], s1)
    assert (torch.cat([o1, o2]) - o).abs().max() < 1e-12 and all((a - b).abs().max() < 1e-12 for a, b in zip(s2, st))


def test_plain_router_chooses_among_the_groups_of_the_best_experts():
    z = torch.log(torch.tensor([[0.30, 0.01, 0.20, 0.19, 0.25, 0.05]], dtype=F64))
    r = dict(experts=6, top=3, groups=dict(count=3, keep=2))
    h, w = torch.ones(1, 1, dtype=F64), z.T.contiguous()
    idx, wt = plain.route(h, w, r)                  # the groups of 0.30 and 0.25; 0.20 and 0.19 are out
    assert idx.tolist() == [[0, 4, 5]] and (wt - torch.tensor([[0.30, 0.25, 0.05]], dtype=F64) / 0.6).abs().max() < 1e-12
    assert plain.route(h, w, dict(experts=6, top=3))[0].tolist() == [[0, 4, 2]]
    # a close call between groups is followed, a far one is refused
    close = torch.tensor([[0.0, -3.0, 1.0, -3.0, 0.99, -2.0]], dtype=F64)
    r = dict(experts=6, top=2, groups=dict(count=3, keep=1))
    idx, wt = plain.route(h, close.T.contiguous(), r)
    assert sorted(idx[0].tolist()) == [2, 3]
    got, _ = plain.follow_close_calls(h, close.T.contiguous(), r, idx, wt, torch.tensor([[4, 5]]), 0.05)
    assert sorted(got[0].tolist()) == [4, 5]
    with pytest.raises(AssertionError):
        plain.follow_close_calls(h, close.T.contiguous(), r, idx, wt, torch.tensor([[0, 1]]), 0.05)
