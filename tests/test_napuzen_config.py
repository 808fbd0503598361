"""The Napuzen configuration reader, its plan and the plain implementation's pieces at hand-computed points (CPU)."""
import copy
import math

import pytest
import torch

import plain_napuzen as plain
from napuzen_models import TINY_N
from xinfer_b200.config import ConfigError, config_from_dict
from xinfer_b200.config.napuzen import SWISH_ALPHA, NapuzenConfig
from xinfer_b200.models.decoder import model_weight_specs
from xinfer_b200.parts.rope import inv_frequencies

F64 = torch.float64


def _plan(cfg):
    entry, c = config_from_dict(cfg)
    assert isinstance(c, NapuzenConfig)
    return entry.plan_of(c)


@pytest.mark.parametrize("name", sorted(TINY_N))
def test_every_key_reaches_a_spec(name):
    cfg = TINY_N[name][0]
    plan = _plan(cfg)
    assert plan.vocab_size == cfg["vocab"] and plan.hidden == cfg["width"] and plan.head_name is None
    assert plan.residual_dtype == "float32" and plan.logit_scale == cfg["logit_scale"]
    assert plan.final_norm.eps == cfg["norm"]["eps"]
    for i, (layer, block, run) in enumerate(zip(cfg["layers"], plan.blocks, plan.runs)):
        m, conv = layer["mixer"], block.mixer
        assert conv.kind == "input_conv" and conv.taps == cfg["canon"]["taps"] and run.block == i
        # the sublayers read the stream itself, the norms stand behind them
        first = block.program[0]
        assert (first.op, first.src) == ("mixer", "x")
        assert [o.name for o in block.program if o.op == "norm"] == (["norm1"] if layer["mlp"] is None else ["norm1", "stream", "norm2"])
        assert all(n.eps == cfg["norm"]["eps"] for n in block.norms() if n.kind == "rmsnorm")
        a = conv.inner
        if layer["type"] == "gla":
            assert (a.heads, a.head_dim, a.v_head_dim, a.tau, a.eps) == (m["heads"], m["dim"], m["vdim"], m["tau"], cfg["norm"]["eps"])
        else:
            assert (a.num_heads, a.head_dim, a.v_head_dim, a.kv_rank, a.scale) == (m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["scale"])
            assert a.norm_eps == cfg["norm"]["eps"] and not a.sink
        if layer["type"] == "latent_attention":
            rot = m["rot"]
            assert a.window is None and not a.gate and a.q_rank == m["q_rank"] and a.rope_dim == m["rot_dim"]
            assert (a.rope.rotary_dim, a.rope.theta, a.rope.layout) == (rot["dims"], rot["base"], "interleaved")
            sc = rot.get("scaling")
            assert a.rope.magnitude == (0.1 * math.log(sc["factor"]) + 1.0 if sc else 1.0)
        elif layer["type"] == "latent_attention_2":
            assert a.window == m["mask"]["size"] and a.gate and a.gate_per_head and a.rope is None and a.rope_dim == 0
            assert a.shares_cache == ("kv_from" in m) and run.cache_from == m.get("kv_from") and a.q_rank is None
        f = block.feed_forward
        if layer["mlp"] is None:
            assert f is None
        elif layer["mlp"]["kind"] == "dense":
            assert (f.kind, f.activation, f.intermediate) == ("swiglu", "swish_clamp", layer["mlp"]["ff"])
            assert f.act_params == (layer["mlp"]["limit"], SWISH_ALPHA)
        else:
            r, sh = layer["mlp"]["router"], layer["mlp"].get("shared")
            assert (f.experts, f.top, f.weight_scale, f.score) == (r["experts"], r["top"], r["scale"], "softmax")
            assert f.renormalize and not f.correction and f.activation == "silu" and f.intermediate == layer["mlp"]["expert"]["ff"]
            assert (f.shared is None) == (sh is None) == (f.shared_gate is None)
            if sh:
                assert f.shared.intermediate == sh["ff"]


def test_cached_rows_are_kept_as_long_as_their_widest_reader_asks():
    def of(name):
        return [b.mixer.inner for b in _plan(TINY_N[name][0]).blocks]
    n1 = of("N1")
    assert n1[1].cache_window == n1[4].cache_window == 37 and n1[1].window == 11     # the reader sees further back
    n2 = of("N2")
    assert [n2[i].cache_window for i in (2, 3, 4)] == [130, 130, 130] and n2[0].cache_window is None
    n3 = of("N3")
    # rows of a layer with a rotated part and no window: the reader masks with its own and skips the rotated channels
    assert n3[2].cache_window is None and n3[2].window == 64 and n3[2].row_tail == 8 and n3[0].row_tail == 0


def test_declared_tensors():
    names = {s.name: tuple(s.shape) for s in model_weight_specs(_plan(TINY_N["N1"][0]))}
    assert names["embed"] == (83, 48) and names["final.norm"] == (48,) and "head" not in names
    assert all(names[f"l{i}.canon1"] == (48, 4) and names[f"l{i}.norm1"] == (48,) for i in range(5))
    assert names["l0.mix.q"] == (30, 48) and names["l0.mix.v"] == (42, 48) and names["l0.mix.g"] == (42, 48)
    assert names["l0.mix.norm"] == (14,) and names["l0.mix.a1"] == (-1, 48) and names["l0.mix.a2"] == (30, -1)
    assert names["l0.mix.a2.b"] == (30,) and names["l0.mix.o"] == (48, 42)
    assert names["l1.mix.q"] == (36, 48) and names["l1.mix.dkv"] == (20, 48) and names["l1.mix.g"] == (3, 48)
    assert names["l1.mix.uk"] == (36, 20) and names["l1.mix.uv"] == (30, 20)
    assert "l4.mix.dkv" not in names and "l4.mix.dkv.norm" not in names and names["l4.mix.uk"] == (18, 20)
    assert names["l3.mix.dq"] == (18, 48) and names["l3.mix.dq.norm"] == (18,) and names["l3.mix.uq"] == (50, 18)
    assert names["l3.mix.dkv"] == (18, 48) and names["l3.mix.dkv.norm"] == (14,) and "l3.mix.q" not in names
    assert names["l0.mlp.router"] == (5, 48) and names["l0.mlp.shared.sg"] == (1, 48) and names["l0.mlp.e4.down"] == (48, 24)
    assert not any(n.startswith("l2.mlp") or n == "l2.norm2" for n in names) and names["l1.mlp.gate"] == (40, 48)


def test_named_errors():
    base = TINY_N["N1"][0]

    def broken(change):
        cfg = copy.deepcopy(base)
        change(cfg)
        with pytest.raises(ConfigError) as e:
            config_from_dict(cfg)
        return str(e.value)

    assert "canon" in broken(lambda c: c.pop("canon"))
    assert "canon.taps" in broken(lambda c: c["canon"].update(taps=0))
    assert "logit_scale" in broken(lambda c: c.pop("logit_scale"))
    assert "layers[0].mixer.tau" in broken(lambda c: c["layers"][0]["mixer"].update(tau=0))
    assert "layers[1].mixer.mask" in broken(lambda c: c["layers"][1]["mixer"].pop("mask"))
    assert "layers[3].mixer.q_rank" in broken(lambda c: c["layers"][3]["mixer"].pop("q_rank"))
    assert "layers[3].mixer.rot.dims" in broken(lambda c: c["layers"][3]["mixer"]["rot"].update(dims=6))
    assert "kv_from" in broken(lambda c: c["layers"][4]["mixer"].update(kv_from=0))          # no latent layer
    assert "kv_rank" in broken(lambda c: c["layers"][4]["mixer"].update(kv_from=3))          # another rank
    assert "kv_from" in broken(lambda c: c["layers"][1]["mixer"].update(kv_from=4))          # not earlier
    assert "layers[2].type" in broken(lambda c: c["layers"][2].update(type="mamba"))
    assert "layers[0].mlp.router.top" in broken(lambda c: c["layers"][0]["mlp"]["router"].update(top=6))
    assert "layers[0].mlp.router.scale" in broken(lambda c: c["layers"][0]["mlp"]["router"].pop("scale"))
    assert "layers[1].mlp.limit" in broken(lambda c: c["layers"][1]["mlp"].update(limit=-1))
    assert "layers[1].mlp.kind" in broken(lambda c: c["layers"][1]["mlp"].update(kind="sparse"))


@pytest.mark.parametrize("dims,base,scaling", [(16, 500.0, None), (8, 30000.0, dict(factor=4.0, original=96, fast=16.0, slow=1.0)),
                                               (32, 1e6, dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
                                               (4, 50.0, dict(factor=3.0, original=64, fast=4.0, slow=0.5))])
def test_frequencies_of_the_product_equal_the_plain_ones(dims, base, scaling):
    from xinfer_b200.config.plan import YarnScaling
    want, _ = plain.yarn_frequencies(dims, base, scaling)
    got = torch.from_numpy(inv_frequencies(base, dims, YarnScaling(**scaling) if scaling else None, True))
    assert ((got.double() - want).abs() <= 1e-6 * want).all()


def test_plain_pieces_at_hand_computed_points():
    # the convolution: zeros before the start, the last tap weighs the token itself
    x = torch.tensor([[1.0], [2.0], [5.0]], dtype=F64)
    assert plain.causal_conv(x, torch.tensor([[10.0, 100.0]], dtype=F64)).flatten().tolist() == [100.0, 210.0, 520.0]
    # the recurrence: the decay acts on key channels, the read sees the token's own write
    q = torch.tensor([[[1.0, 0.0]], [[1.0, 1.0]]], dtype=F64)
    k = torch.tensor([[[2.0, 3.0]], [[0.0, 1.0]]], dtype=F64)
    v = torch.tensor([[[4.0]], [[7.0]]], dtype=F64)
    alpha = torch.tensor([[[0.9, 0.9]], [[0.5, 0.25]]], dtype=F64)
    o, S = plain.linear_recurrence(q, k, v, alpha)
    assert o.flatten().tolist() == [8.0, 0.5 * 8.0 + 0.25 * 12.0 + 7.0] and S.flatten().tolist() == [4.0, 10.0]
    assert abs(float(plain.key_decay(torch.tensor(0.0, dtype=F64), 2.0)) - math.sqrt(0.5)) < 1e-15
    # a quarter turn of the first pair, magnitude of the stretch
    rot = dict(dims=2, base=10.0)
    y = plain.rotate_neighbours(torch.tensor([[[3.0, 4.0, 9.0]]], dtype=F64), torch.tensor([math.pi / 2]), rot)
    assert (y - torch.tensor([[[-4.0, 3.0, 9.0]]], dtype=F64)).abs().max() < 1e-6
    # the window counts the token itself
    assert plain.causal_mask(4, 2)[3].tolist() == [False, False, True, True] and plain.causal_mask(3)[2].all()
    # the router's weights are a softmax over all experts, renormalized over the chosen ones
    h, wr = torch.tensor([[1.0]], dtype=F64), torch.tensor([[0.0], [math.log(3.0)], [math.log(2.0)]], dtype=F64)
    idx, wt = plain.route(h, wr, 2, 2.0)
    assert idx.tolist() == [[1, 2]] and (wt - torch.tensor([[1.2, 0.8]], dtype=F64)).abs().max() < 1e-12


def test_plain_cuts_agree():
    """The plain recurrence carried over a cut equals the whole (the oracle of the scans' tests)."""
    g = torch.Generator().manual_seed(1)
    q, k, v, a = (torch.randn(9, 2, d, generator=g, dtype=F64) for d in (3, 3, 4, 3))
    a = torch.sigmoid(a)
    o, S = plain.linear_recurrence(q, k, v, a)
    o1, S1 = plain.linear_recurrence(q[:4], k[:4], v[:4], a[:4])
    o2, S2 = plain.linear_recurrence(q[4:], k[4:], v[4:], a[4:], S1)
    assert (torch.cat([o1, o2]) - o).abs().max() < 1e-12 and (S2 - S).abs().max() < 1e-12
