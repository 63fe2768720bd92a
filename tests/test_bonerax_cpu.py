"""Bonerax without a GPU: configuration, registry, tensor names, what the cache manager is asked for, the plain model's
mechanisms against properties that follow from their definitions, and the engine's own step function, cache and state
manager and replay program over plain statements of the kernels against the plain model."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_bonerax as pb
import plain_ops
import tiny
import tiny_bonerax as tb
import traces
from fastmlx_b200 import registry
from fastmlx_b200.config import ConfigError, YarnScaling
from fastmlx_b200.config.bonerax import BoneraxConfig
from fastmlx_b200.parts import (ChannelDeltaMixer, FreeDim, GatedLinearAttention, GQAAttention, LayerNorm, PagedKVSpec, PairMixer,
                                PostNormBlock, RoutedExperts, SwiGLU, inverse_frequencies)


def test_registry_finds_the_design_and_builds_its_layers():
    cfg, model = registry.build_model(tb.B1)
    assert isinstance(cfg, BoneraxConfig) and cfg.vocab_size == 211 and cfg.width == 96 and cfg.norm_eps == 1e-6
    assert cfg.logit_scale == 0.7 and cfg.logit_softcap == 11.0 and model.head.scale == 0.7 and model.head.softcap == 11.0
    assert len(model.layers) == 4 and [r.layer for r in model.schedule] == [0, 1, 2, 0, 2, 3]
    assert all(isinstance(b, PostNormBlock) and isinstance(b.norm1, LayerNorm) for b in model.layers)
    assert [type(b.mixer) for b in model.layers] == [PairMixer, GatedLinearAttention, ChannelDeltaMixer, GatedLinearAttention]
    assert [type(b.ffn) for b in model.layers] == [RoutedExperts, RoutedExperts, SwiGLU, type(None)]
    a, d = model.layers[0].mixer.left, model.layers[0].mixer.right
    assert isinstance(a, GQAAttention) and isinstance(d, ChannelDeltaMixer) and a.general and a.late_bias and a.o is None and d.o is None
    assert (a.nh, a.nkv, a.hd, a.vd, a.scale, a.window, a.value_scale, d.out_scale) == (4, 2, 16, 32, 0.3, 19, 1.25, -0.6)
    assert a.qk_norm_first and not a.qk_norm_whole and a.pos.traditional and a.pos.rotary_dim == 8
    assert a.pos.scaling == YarnScaling(4.0, 96.0, 8.0, 1.5) and a.pos.amplitude == pytest.approx(0.1 * math.log(4.0) + 1.0)
    assert (d.H, d.G, d.D, d.Dv, d.taps) == (4, 2, 12, 20, 3)
    e = model.layers[0].ffn
    assert (e.E, e.top, e.ff, e.activation, e.renorm, e.shared_ff, e.router_bias_name) == (6, 2, 24, "silu", True, 0, "l0.mlp.router.b")
    assert model.layers[3].mixer.tau == 1.0
    _, plain = registry.build_model(tb.B2)
    assert plain.head.scale == 1.0 and plain.head.softcap == 0.0
    assert plain.layers[2].mixer.left.window == 0 and plain.layers[2].mixer.left.pos.amplitude == 1.0


def test_every_run_of_a_shared_layer_has_pages_and_a_state_of_its_own():
    _, model = registry.build_model(tb.B1)
    needs = model.cache_needs()
    assert len(needs) == 6 and all(src is None for _, _, src in needs)
    assert needs[0][0] == needs[3][0] == PagedKVSpec(2, 16, 19, 32) and all(needs[i][0] is None for i in (1, 2, 4, 5))
    floats = {0: 4 * 20 * 12 + 2 * (2 * 2 * 12 + 4 * 20), 1: 3 * 12 * 20, 2: 6 * 16 * 24 + 3 * (2 * 2 * 24 + 6 * 16), 5: 2 * 40 * 8}
    for i, n in floats.items():
        assert needs[i][1].dtype == torch.float32 and n <= needs[i][1].shape[0] < n + 4 and needs[i][1].shape[0] % 4 == 0
    assert needs[3][1] == needs[0][1] and needs[4][1] == needs[2][1] and model.graph_safe
    from fastmlx_b200.cache.manager import CacheManager
    m = CacheManager(needs, page_size=8, num_pages=16, max_requests=2, dtype=torch.float32)
    assert m.entries[0].kv.data_ptr() != m.entries[3].kv.data_ptr() and m.entries[0].state.data_ptr() != m.entries[3].state.data_ptr()


def test_a_model_without_pages_is_never_short_of_them():
    from fastmlx_b200.cache.manager import CacheManager
    _, model = registry.build_model(tb.one_layer("gla", tb.gla(2, 8, 8, 2.0)))
    m = CacheManager(model.cache_needs(), page_size=8, num_pages=1, max_requests=2, dtype=torch.float32)
    r = m.add_request("a")
    assert m.pages_needed(r, 1000) == 0 and m.free_pages > 1000 and m.holds_alone(10 ** 6, 512) == 0
    m.reserve(r, 1000)
    m.commit(r)
    m.check()
    m.free("a")


def test_tensor_names_and_shapes():
    _, model = registry.build_model(tb.B1)
    specs = {s.name: tuple(s.shape) for s in model.weight_specs()}
    assert specs["embed"] == (211, 96) and specs["head"] == (211, 96) and specs["final.norm"] == (96,)
    assert specs["l0.mix.left.q"] == (64, 96) and specs["l0.mix.left.k"] == (32, 96) and specs["l0.mix.left.v"] == (64, 96)
    assert specs["l0.mix.left.q.b"] == (64,) and specs["l0.mix.left.v.b"] == (64,) and specs["l0.mix.left.o.b"] == (96,)
    assert specs["l0.mix.left.q.norm"] == specs["l0.mix.left.k.norm"] == (16,) and specs["l0.mix.left.o"] == (96, 128)
    assert specs["l0.mix.right.q"] == specs["l0.mix.right.k"] == (24, 96) and specs["l0.mix.right.v"] == (80, 96)
    assert specs["l0.mix.right.k.conv"] == (24, 3) and specs["l0.mix.right.v.conv"] == (80, 3)
    assert specs["l0.mix.right.A_log"] == (4,) and specs["l0.mix.right.dt_bias"] == (48,) and specs["l0.mix.right.norm"] == (20,)
    assert specs["l0.mix.right.a2"][0] == 48 and specs["l0.mix.right.g2"][0] == 80 and specs["l0.mix.right.b"] == (4, 96)
    assert specs["l0.mix.right.o"] == (96, 80)
    assert specs["l1.mix.q"] == specs["l1.mix.k"] == (60, 96) and specs["l1.mix.v"] == specs["l1.mix.g"] == (36, 96)
    assert specs["l1.mix.a2.b"] == (60,) and specs["l1.mix.norm"] == (12,) and specs["l1.mix.o"] == (96, 36)
    assert specs["l0.mlp.router"] == (6, 96) and specs["l0.mlp.router.b"] == (6,) and specs["l0.mlp.e5.down"] == (96, 24)
    assert specs["l2.mlp.gate"] == (96, 96) and "l5.norm2" not in specs
    assert not any(n.startswith(("l3.", "l4.", "l5.mlp")) for n in specs)
    tensors = tb.lively_tensors(tb.B1, 3)
    model.check_weights(tensors)
    model.check_weights(dict(tensors, **{"l5.norm2": torch.ones(96)}))
    with pytest.raises(Exception):
        model.check_weights({k: v for k, v in tensors.items() if k != "l0.mlp.router.b"})


def test_ranks_come_from_the_tensors_and_must_agree():
    from fastmlx_b200.weights.loader import WeightError
    _, model = registry.build_model(tb.B1)
    spec = {s.name: s for s in model.weight_specs()}
    assert isinstance(spec["l1.mix.a1"].shape[0], FreeDim) and isinstance(spec["l1.mix.a2"].shape[1], FreeDim)
    tensors = tb.lively_tensors(tb.B1, 3)
    assert tensors["l1.mix.a1"].shape == (8, 96) and tensors["l0.mix.right.g2"].shape == (80, 24)
    bad = dict(tensors, **{"l1.mix.a2": torch.zeros(60, 7, dtype=torch.bfloat16)})
    with pytest.raises(WeightError) as err:
        model.check_weights(bad)
    assert [w[0] for w in err.value.wrong_shape] == ["l1.mix.a2"]
    # the random initialiser uses the parts' own ranks, and they agree with one another
    from fastmlx_b200.weights.random_init import random_tensors
    r = random_tensors(model, 1)
    model.check_weights(r)


@pytest.mark.parametrize("breakage", [
    lambda c: c["layers"][0].update(type="serial"),
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["right"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=18),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"].pop("right_scale"),
    lambda c: c["layers"][0]["mixer"].pop("right"),
    lambda c: c["layers"][1]["mixer"].update(tau=0),
    lambda c: c["layers"][2]["mixer"].update(conv=17),
    lambda c: c["layers"][3].update(weights_of=9),
    lambda c: c["layers"][3].update(weights_of=2),
    lambda c: c["layers"][0].update(weights_of=3),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][0]["mlp"].pop("expert"),
    lambda c: c.pop("norm"),
    lambda c: c.update(logit_softcap=-1.0),
    lambda c: c.update(layers=[]),
])
def test_bad_configurations_are_refused(breakage):
    cfg = copy.deepcopy(tb.B1)
    breakage(cfg)
    with pytest.raises(ConfigError):
        BoneraxConfig.from_dict(cfg)


@pytest.mark.parametrize("dims,base,scaling", [(8, 500.0, (4.0, 96, 8.0, 1.5)), (64, 250000.0, (3.0, 128, 16.0, 1.0)), (6, 777.0, (2.0, 40, 6.0, 1.0)),
                                               (32, 10000.0, (16.0, 4096, 32.0, 1.0)), (16, 20.0, (2.0, 8, 64.0, 32.0))])
def test_yarn_frequencies_of_the_part_are_those_of_the_plain_model(dims, base, scaling):
    f, mult = pb.yarn(tb.rot(dims, base, scaling))
    y = YarnScaling(*(float(s) for s in scaling))
    got = inverse_frequencies(dims, base, y)
    assert torch.allclose(got, torch.tensor(f, dtype=torch.float64), rtol=1e-12, atol=0) and y.amplitude == pytest.approx(mult)


# ---- the plain model's mechanisms
def _weights(shapes, seed, scale=0.5):
    g = torch.Generator().manual_seed(seed)
    return {n: torch.randn(*s, generator=g, dtype=torch.float64) * scale for n, s in shapes.items()}, g


def test_plain_yarn_keeps_fast_pairs_and_slows_slow_ones():
    plain, one = pb.yarn(tb.rot(64, 10000.0))
    f, mult = pb.yarn(tb.rot(64, 10000.0, (8.0, 2048, 32.0, 1.0)))
    assert one == 1.0 and mult == pytest.approx(0.1 * math.log(8.0) + 1.0)
    turns = [2048 * p / (2 * math.pi) for p in plain]                 # how often a pair turns within the original length
    for p, q, n in zip(plain, f, turns):
        if n > 40:
            assert q == p
        if n < 0.8:
            assert q == pytest.approx(p / 8.0)
        assert p / 8.0 * (1 - 1e-12) <= q <= p
    assert any(p / 8.0 < q < p for p, q in zip(plain, f))


def test_plain_rotation_pairs_neighbours_and_scales_what_it_turns():
    u = torch.zeros(3, 1, 10, dtype=torch.float64)
    u[:, 0, 2] = 1.0
    u[:, 0, 9] = 5.0
    r = tb.rot(6, 100.0, (2.0, 50, 4.0, 1.0))
    f, mult = pb.yarn(r)
    out = pb.rotate(u, r)
    for p in range(3):
        assert float(out[p, 0, 2]) == pytest.approx(mult * math.cos(p * f[1]))
        assert float(out[p, 0, 3]) == pytest.approx(mult * math.sin(p * f[1]))
        assert float(out[p, 0, 9]) == 5.0 and float(out[p, 0, 4]) == 0.0


def test_plain_window_holds_the_token_and_those_just_before_it():
    m = tb.attention(1, 1, 2, 3, 1.0, window=3)
    T, width = 8, 4
    W, g = _weights({"q": (2, width), "k": (2, width), "v": (3, width), "q.b": (2,), "k.b": (2,), "v.b": (3,)}, 1)
    W.update({"q.norm": torch.ones(2, dtype=torch.float64), "k.norm": torch.ones(2, dtype=torch.float64),
              "o": torch.eye(3, dtype=torch.float64), "o.b": torch.zeros(3, dtype=torch.float64)})
    h = torch.randn(T, width, generator=g, dtype=torch.float64)
    y = pb.windowed_attention(h, W, m, 1e-6)
    for j in range(T):
        h2 = h.clone()
        h2[j] += 1.0
        moved = (pb.windowed_attention(h2, W, m, 1e-6) - y).abs().max(dim=1).values > 1e-9
        assert moved.tolist() == [j <= i < j + 3 for i in range(T)]


def test_plain_delta_rule_replaces_what_a_key_stored():
    """With decays of one and write strengths of one, reading a unit key right after writing to it gives the value just
    written, whatever the key held before."""
    H, D, Dv = 1, 3, 2
    m = tb.delta(H, H, D, Dv, 1)
    W, g = _weights({"q": (3, 5), "k": (3, 5), "v": (2, 5), "b": (1, 5), "a1": (2, 5), "g1": (2, 5)}, 3)
    ones = lambda *s: torch.ones(*s, dtype=torch.float64)
    W.update({"q": W["k"], "q.conv": ones(3, 1), "k.conv": ones(3, 1), "v.conv": ones(2, 1), "A_log": ones(1) * -60.0,
              "a2": torch.zeros(3, 2, dtype=torch.float64), "dt_bias": torch.zeros(3, dtype=torch.float64),
              "g2": torch.zeros(2, 2, dtype=torch.float64), "norm": ones(2), "o": torch.eye(2, dtype=torch.float64)})
    h = torch.randn(6, 5, generator=g, dtype=torch.float64)
    W["b"] = W["b"] * 0.0
    h[:, 0] = 1.0
    W["b"][0, 0] = 60.0
    y = pb.channel_delta(h, W, m, 0.0)
    v = pb.silu(h @ W["v"].T)
    assert torch.allclose(y, 0.5 * pb.rms_norm(v, 0.0), atol=1e-4)          # sigmoid(0) gates by a half


def test_plain_gated_linear_attention_equals_its_sum_over_earlier_tokens():
    m = tb.gla(2, 3, 4, 2.5)
    T, width = 7, 5
    W, g = _weights({"q": (6, width), "k": (6, width), "v": (8, width), "g": (8, width), "a1": (2, width), "a2": (6, 2), "a2.b": (6,)}, 2)
    W.update({"norm": torch.ones(4, dtype=torch.float64), "o": torch.eye(8, dtype=torch.float64)})
    h = torch.randn(T, width, generator=g, dtype=torch.float64)
    y = pb.gated_linear_attention(h, W, m, 1e-6)
    q, k, v = (h @ W["q"].T).reshape(T, 2, 3) * 3 ** -0.5, (h @ W["k"].T).reshape(T, 2, 3), (h @ W["v"].T).reshape(T, 2, 4)
    a = (torch.sigmoid((h @ W["a1"].T) @ W["a2"].T + W["a2.b"]) ** 0.4).reshape(T, 2, 3)
    o = torch.zeros(T, 2, 4, dtype=torch.float64)
    for t in range(T):
        for s in range(t + 1):
            decay = a[s + 1:t + 1].prod(0)
            o[t] += torch.einsum("hd,hv->hv", q[t] * k[s] * decay, v[s])
    assert torch.allclose(y, pb.rms_norm(o, 1e-6).reshape(T, 8) * pb.silu(h @ W["g"].T), atol=1e-10)


def test_plain_router_weighs_by_the_chosen_logits_alone():
    mlp = tb.moe(4, 2, 3)
    width = 5
    W, g = _weights({f"e{e}.{n}": s for e in range(4) for n, s in (("gate", (3, width)), ("up", (3, width)), ("down", (width, 3)))}, 3)
    W.update(_weights({"router": (4, width)}, 4)[0])
    h = torch.randn(1, width, generator=g, dtype=torch.float64)
    z = (h @ W["router"].T)[0]
    W["router.b"] = torch.zeros(4, dtype=torch.float64)
    order = torch.argsort(z, descending=True).tolist()
    W["router.b"][order[3]] = float(z[order[0]] - z[order[3]]) + 1.0          # a bias that lifts the weakest above all others
    y = pb.routed_feed_forward(h, W, mlp)
    e = math.e
    want = e / (1 + e) * pb.gated(h, pb.sub(W, f"e{order[3]}.")) + 1 / (1 + e) * pb.gated(h, pb.sub(W, f"e{order[0]}."))
    assert torch.allclose(y, want, atol=1e-12)


def test_plain_layer_norm_and_capped_logits():
    x = torch.tensor([[1.0, 2.0, 6.0]], dtype=torch.float64)
    w = torch.tensor([1.0, 2.0, 3.0], dtype=torch.float64)
    sd = math.sqrt((4 + 1 + 9) / 3 + 0.5)
    assert torch.allclose(pb.layer_norm(x, 0.5, w), torch.tensor([[-2.0, -2.0, 9.0]], dtype=torch.float64) / sd)
    W = {"final.norm": w, "head": torch.eye(3, dtype=torch.float64)}
    raw = pb.output(x, W, {"logit_scale": 3.0}, 0.5)
    assert torch.allclose(pb.output(x, W, {"logit_scale": 3.0, "logit_softcap": 2.0}, 0.5), 2.0 * torch.tanh(raw / 2.0))


def test_plain_forward_is_causal_and_shared_layers_keep_states_apart():
    W = {n: t.double() for n, t in tb.lively_tensors(tb.B1, 5).items()}
    toks = tiny.rand_tokens(40, 211, 1)
    full, streams = pb.forward(tb.B1, W, toks, return_layers=True)
    assert streams.shape == (6, 40, 96)
    assert torch.allclose(pb.forward(tb.B1, W, toks[:17]), full[:17], atol=1e-10)
    # the same model with copies of the shared tensors under names of their own
    cfg = copy.deepcopy(tb.B1)
    for i, j in ((3, 0), (4, 2)):
        del cfg["layers"][i]["weights_of"]
        W.update({f"l{i}." + n[len(f"l{j}."):]: t for n, t in list(W.items()) if n.startswith(f"l{j}.")})
    assert torch.equal(pb.forward(cfg, W, toks), full)


# ---- the engine over plain statements of the kernels
LENS = {"B1": [1, 2, 9, 45, 58], "B2": [3, 50, 65], "B3": [5, 40, 90], "B4": [4, 41, 60]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bonerax_cpu")
    out = {}
    for name, cfg in tb.CONFIGS.items():
        d = tb.make_model_dir(root, cfg, seed=11)
        W = tiny.load_plain_weights(d)
        prompts = {f"r{i}": tiny.rand_tokens(n, cfg["vocab"], 500 + i) for i, n in enumerate(LENS[name])}
        out[name] = (d, prompts, {r: pb.forward(cfg, W, t) for r, t in prompts.items()})
    return out


@pytest.mark.parametrize("name", ["B1", "B2", "B3", "B4"])
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed"])
def test_engine_over_plain_kernels_matches_the_plain_model(models, name, cut):
    from fastmlx_b200.engine.replay import Replayer
    d, prompts, ref = models[name]
    steps = {"whole": traces.whole, "tail": lambda p: traces.tail_decoded(p, tail=12), "portions": traces.portions,
             "mixed": lambda p: traces.mixed(p, max_live=2)}[cut](prompts)
    rp = Replayer(d, "float32", 192, page_size=8, device="cpu", kernels=plain_ops, max_live=2)
    outs = []
    for st in steps:
        outs.append(rp.step(st))
        rp.manager.check()
    assert not rp.manager.requests and all(g.pool.used_pages == 0 for g in rp.manager.groups)
    rows = traces.collect(steps, outs)
    for rid, toks in prompts.items():
        got = torch.from_numpy(np.stack([rows[rid][i] for i in range(len(toks))])).double()
        err = (got - ref[rid]).abs().max() / ref[rid].abs().max()
        assert err < 3e-5, (rid, float(err))
