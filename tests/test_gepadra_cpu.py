"""Gepadra without a GPU: configuration, registry, tensor names, what the cache manager is asked for, the plain model's
mechanisms against properties that follow from their definitions, and the engine's own step function, cache and state
manager and replay program over plain statements of the kernels against the plain model."""
import copy
import math

import numpy as np
import pytest
import torch

import plain_gepadra as pg
import plain_ops
import tiny
import tiny_gepadra as tg
import traces
from fastmlx_b200 import registry
from fastmlx_b200.config import ConfigError, GepadraConfig
from fastmlx_b200.parts import (GQAAttention, MatrixMemoryMixer, PagedKVSpec, ParallelBlock, PlainRoutedExperts, RMSNorm, SwiGLU)


def test_registry_finds_the_design_and_builds_its_layers():
    cfg, model = registry.build_model(tg.G1)
    assert isinstance(cfg, GepadraConfig) and cfg.vocab_size == 211 and cfg.width == 96 and cfg.norm_eps == 1e-6 and cfg.first_v_mix == 1
    assert all(isinstance(b, ParallelBlock) and isinstance(b.norm, RMSNorm) and b.norm.offset == 1.0 for b in model.layers)
    assert [type(b.mixer) for b in model.layers] == [MatrixMemoryMixer, GQAAttention, MatrixMemoryMixer, GQAAttention, GQAAttention, MatrixMemoryMixer]
    assert [type(b.ffn) for b in model.layers] == [PlainRoutedExperts, SwiGLU, type(None), PlainRoutedExperts, type(None), SwiGLU]
    assert [b.norm2 is None for b in model.layers] == [False, False, True, False, True, False]
    a = model.layers[1].mixer
    assert (a.nh, a.nkv, a.hd, a.vd, a.scale, a.window, a.keep_first, a.value_mix) == (4, 2, 16, 32, 0.3, 19, 5, "first")
    assert a.general and a.qk_norm_eps is None and not a.pos.traditional and a.pos.rotary_dim == 8 and a.o is None and not a.late_bias
    assert [model.layers[i].mixer.value_mix for i in (3, 4)] == ["later", "later"] and model.layers[4].mixer.window == 0
    m = model.layers[0].mixer
    assert (m.H, m.D, m.Dv, m.cap, m.o) == (3, 20, 12, 6.0, None)
    e = model.layers[0].ffn
    assert (e.E, e.top, e.ff, e.shared_ff, e.activation, e.scores, e.weigh, e.scale) == (6, 2, 24, 40, "gelu", "sigmoid", "input", 1.0)
    assert model.layers[3].ffn.shared_ff == 0 and model.layers[3].ffn.gate_name is None
    assert model.layers[1].ffn.limit == 0.9 and model.head.tied is model.embed
    # the joined output product takes the mixer's heads, every expert's and the shared expert's hidden layer
    assert model.layers[0].out.in_features == 3 * 12 + 6 * 24 + 40 and model.layers[2].out.in_features == 2 * 40
    _, other = registry.build_model(tg.G2)
    assert [other.layers[i].mixer.value_mix for i in (0, 2)] == ["first", None] and other.layers[0].mixer.pos.native_args()[0] is None


def test_pages_and_state_slots():
    _, model = registry.build_model(tg.G1)
    needs = model.cache_needs()
    assert [n[0] for n in needs] == [None, PagedKVSpec(2, 16, 19, 32, 5), None, PagedKVSpec(2, 24, 11, 32, 21), PagedKVSpec(4, 16, 0, 0, 0), None]
    for i, (h, d, v) in {0: (3, 20, 12), 2: (2, 8, 40), 5: (4, 16, 24)}.items():
        n = h * (v + 1) * d + h
        assert needs[i][1].dtype == torch.float32 and n <= needs[i][1].shape[0] < n + 4 and needs[i][1].shape[0] % 4 == 0
    assert model.graph_safe


def test_tensor_names_and_shapes():
    _, model = registry.build_model(tg.G1)
    specs = {s.name: tuple(s.shape) for s in model.weight_specs()}
    assert len(specs) == len(model.weight_specs())
    assert specs["embed"] == (211, 96) and "head" not in specs and specs["final.norm"] == (96,)
    assert specs["l0.mix.q"] == specs["l0.mix.k"] == (60, 96) and specs["l0.mix.v"] == specs["l0.mix.g"] == (36, 96)
    assert specs["l0.mix.i"] == specs["l0.mix.f"] == (3, 96) and specs["l0.mix.i.b"] == specs["l0.mix.f.b"] == (3,)
    assert specs["l0.mix.norm"] == (36,) and specs["l0.mix.o"] == (96, 36)
    assert specs["l0.mlp.router"] == (6, 96) and specs["l0.mlp.e5.up"] == (24, 96) and specs["l0.mlp.e5.down"] == (96, 24)
    assert specs["l0.mlp.shared.up"] == (40, 96) and specs["l0.mlp.shared.down"] == (96, 40) and specs["l0.mlp.shared.sg"] == (1, 96)
    assert specs["l1.mix.q"] == (64, 96) and specs["l1.mix.k"] == (32, 96) and specs["l1.mix.v"] == (64, 96) and specs["l1.mix.v.b"] == (64,)
    assert specs["l1.mix.sink"] == (4,) and specs["l1.mix.vmix"] == () and specs["l1.mix.o"] == (96, 128) and "l1.mix.o.b" not in specs
    assert specs["l1.mlp.gate"] == specs["l1.mlp.up"] == (96, 96) and "l3.mlp.shared.sg" not in specs and "l2.norm2" not in specs
    tensors = tg.lively_tensors(tg.G1, 3)
    model.check_weights(tensors)
    model.check_weights(dict(tensors, **{"l2.norm2": torch.zeros(96)}))
    for name in ("l1.mix.sink", "l1.mix.vmix", "l0.mix.f.b", "l0.mlp.e3.down"):
        with pytest.raises(Exception):
            model.check_weights({k: v for k, v in tensors.items() if k != name})
    _, other = registry.build_model(tg.G2)
    assert "l2.mix.vmix" not in {s.name for s in other.weight_specs()}
    from fastmlx_b200.weights.random_init import random_tensors
    model.check_weights(random_tensors(model, 1))


@pytest.mark.parametrize("breakage", [
    lambda c: c["layers"][0].update(type="lstm"),
    lambda c: c["layers"][0].pop("mixer"),
    lambda c: c["layers"][0]["mixer"].pop("gate_cap"),
    lambda c: c["layers"][0]["mixer"].update(gate_cap=0),
    lambda c: c["layers"][0]["mixer"].update(dim=600),
    lambda c: c["layers"][1]["mixer"].update(kv_heads=3),
    lambda c: c["layers"][1]["mixer"].update(v_mix=1),
    lambda c: c["layers"][1]["mixer"].update(vdim=16),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7),
    lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18),
    lambda c: c["layers"][1]["mixer"]["rot"].update(base=0),
    lambda c: c["layers"][1]["mixer"]["mask"].update(size=0),
    lambda c: c["layers"][1]["mixer"]["mask"].update(keep_first=-1),
    lambda c: c["layers"][1]["mixer"].pop("scale"),
    lambda c: c["layers"][1]["mlp"].pop("limit"),
    lambda c: c["layers"][1]["mlp"].update(limit=-0.5),
    lambda c: c["layers"][0]["mlp"]["router"].update(top=7),
    lambda c: c["layers"][0]["mlp"].update(kind="sparse"),
    lambda c: c["layers"][0]["mlp"].pop("expert"),
    lambda c: c.pop("norm"),
    lambda c: c.update(layers=[]),
])
def test_bad_configurations_are_refused(breakage):
    cfg = copy.deepcopy(tg.G1)
    breakage(cfg)
    with pytest.raises(ConfigError):
        GepadraConfig.from_dict(cfg)


def test_absent_and_null_options_mean_none():
    a, b = copy.deepcopy(tg.G2), copy.deepcopy(tg.G2)
    a["layers"][0]["mixer"].update(mask=None, rot=None)
    for i in (0, 2):
        b["layers"][i]["mixer"].pop("v_mix")
    a["layers"][1]["mlp"] = None
    del b["layers"][1]["mlp"]
    ca, cb = GepadraConfig.from_dict(a), GepadraConfig.from_dict(b)
    assert ca.layers[0].mixer.window == 0 and ca.layers[0].mixer.rot_dims == 0 and ca.layers[1].mlp is None and cb.layers[1].mlp is None
    assert not cb.layers[0].mixer.v_mix and cb.first_v_mix is None and ca.first_v_mix == 0 and ca.to_dict() == a


# ---- the plain model's mechanisms
def _rand(shapes, seed, scale=0.5):
    g = torch.Generator().manual_seed(seed)
    return {n: torch.randn(*s, generator=g, dtype=torch.float64) * scale for n, s in shapes.items()}, g


def _attention_weights(H, G, D, Dv, width, seed):
    W, g = _rand({"q": (H * D, width), "k": (G * D, width), "v": (G * Dv, width), "q.b": (H * D,), "k.b": (G * D,), "v.b": (G * Dv,), "sink": (H,)}, seed)
    W["o"] = torch.eye(H * Dv, dtype=torch.float64)
    return W, g


def test_plain_window_keeps_the_first_tokens():
    m = tg.attention(1, 1, 2, 3, 1.0, (3, 2))
    W, g = _attention_weights(1, 1, 2, 3, 4, 1)
    h = torch.randn(9, 4, generator=g, dtype=torch.float64)
    y = pg.attention(h, W, m, 1e-6, {})
    for j in range(9):
        h2 = h.clone()
        h2[j] += 1.0
        moved = (pg.attention(h2, W, m, 1e-6, {}) - y).abs().max(dim=1).values > 1e-9
        assert moved.tolist() == [j <= i and (i - j < 3 or j < 2) for i in range(9)]


def test_plain_sink_takes_its_share_once_and_unscaled():
    m = tg.attention(2, 1, 4, 3, 0.3)
    W, g = _attention_weights(2, 1, 4, 3, 6, 2)
    h = torch.randn(5, 6, generator=g, dtype=torch.float64)
    y = pg.attention(h, W, m, 1e-6, {}).reshape(5, 2, 3)
    q, k, v = (h @ W["q"].T + W["q.b"]).reshape(5, 2, 4), h @ W["k"].T + W["k.b"], h @ W["v"].T + W["v.b"]
    for t in range(5):
        for hd in range(2):
            e = torch.exp(0.3 * (k[:t + 1] @ q[t, hd]))
            assert torch.allclose(y[t, hd], (e @ v[:t + 1]) / (e.sum() + torch.exp(W["sink"][hd])), atol=1e-12)


def test_plain_rotation_pairs_halves():
    u = torch.zeros(4, 1, 9, dtype=torch.float64)
    u[:, 0, 1], u[:, 0, 8] = 1.0, 5.0
    out = pg.rotate(u, {"dims": 6, "base": 100.0})
    for p in range(4):
        a = p * 100.0 ** (-2.0 / 6)
        assert float(out[p, 0, 1]) == pytest.approx(math.cos(a)) and float(out[p, 0, 4]) == pytest.approx(math.sin(a))
        assert float(out[p, 0, 8]) == 5.0 and float(out[p, 0, 2]) == 0.0


def test_plain_values_are_mixed_with_the_first_mixing_layers_own():
    """The first mixing layer's values go in as projected (its own share is not used); a later one attends over the mix."""
    m = tg.attention(1, 1, 2, 3, 0.4, v_mix=True)
    W1, g = _attention_weights(1, 1, 2, 3, 4, 3)
    W2, _ = _attention_weights(1, 1, 2, 3, 4, 4)
    W1["vmix"], W2["vmix"] = torch.tensor(0.9, dtype=torch.float64), torch.tensor(0.25, dtype=torch.float64)
    h = torch.randn(6, 4, generator=g, dtype=torch.float64)
    first = {}
    plain = dict(m, v_mix=False)
    assert torch.equal(pg.attention(h, W1, m, 1e-6, first), pg.attention(h, W1, plain, 1e-6, {}))
    y = pg.attention(2 * h, W2, m, 1e-6, first)
    own, other = pg.attention(2 * h, W2, plain, 1e-6, {}), pg.attention(2 * h, dict(W2, v=W1["v"] / 2, **{"v.b": W1["v.b"]}), plain, 1e-6, {})
    assert torch.allclose(y, 0.75 * own + 0.25 * other, atol=1e-12)


def test_plain_memory_equals_its_sum_over_earlier_tokens():
    """Without the running maximum: weights exp(sum of later f + i), and a denominator of at least 1 (exp(-m) scaled back)."""
    H, D, Dv, T = 2, 3, 4, 9
    g = torch.Generator().manual_seed(5)
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, Dv))
    i, f = torch.randn(T, H, generator=g, dtype=torch.float64) * 3, pg.log_sigmoid(torch.randn(T, H, generator=g, dtype=torch.float64) * 3)
    o = pg.mlstm_walk(q, k, v, i, f)
    for t in range(T):
        w = torch.stack([torch.exp(i[s] + f[s + 1:t + 1].sum(0)) for s in range(t + 1)])          # [s, H]
        S = torch.einsum("sh,shd,shv->hdv", w, k[:t + 1], v[:t + 1])
        n = torch.einsum("sh,shd->hd", w, k[:t + 1])
        m = torch.zeros(H, dtype=torch.float64)
        for s in range(t + 1):
            m = torch.maximum(f[s] + m, i[s])
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.ones(H, dtype=torch.float64)) + 1e-6 * torch.exp(m)
        assert torch.allclose(o[t], torch.einsum("hdv,hd->hv", S, q[t]) / den[:, None], rtol=1e-10, atol=1e-12)


def test_plain_gates_are_capped():
    W, g = _rand({"i": (2, 3), "f": (2, 3), "i.b": (2,), "f.b": (2,)}, 6, scale=50.0)
    i, f = pg.log_gates(torch.randn(40, 3, generator=g, dtype=torch.float64), W, 4.0)
    assert float(i.abs().max()) <= 4.0 and float(i.max()) > 3.9 and float(i.min()) < -3.9
    assert float(f.max()) <= -math.log1p(math.exp(-4.0)) + 1e-12 and float(f.min()) >= -math.log1p(math.exp(4.0)) - 1e-12


def test_plain_router_weighs_the_inputs_by_sigmoids():
    mlp = tg.moe(4, 2, 3, 5)
    W, g = _rand({f"e{e}.{n}": s for e in range(4) for n, s in (("up", (3, 6)), ("down", (6, 3)))}, 7)
    W.update(_rand({"router": (4, 6), "shared.up": (5, 6), "shared.down": (6, 5), "shared.sg": (1, 6)}, 8)[0])
    h = torch.randn(1, 6, generator=g, dtype=torch.float64)
    s = torch.sigmoid(h @ W["router"].T)[0]
    a, b = torch.argsort(s, descending=True)[:2].tolist()
    gelu = torch.nn.functional.gelu
    want = sum(gelu((s[e] * h) @ W[f"e{e}.up"].T) @ W[f"e{e}.down"].T for e in (a, b))
    want = want + torch.sigmoid(h @ W["shared.sg"].T) * (gelu(h @ W["shared.up"].T) @ W["shared.down"].T)
    assert torch.allclose(pg.routed(h, W, mlp), want, atol=1e-12)
    outside = sum(s[e] * (gelu(h @ W[f"e{e}.up"].T) @ W[f"e{e}.down"].T) for e in (a, b))
    assert not torch.allclose(outside, sum(gelu((s[e] * h) @ W[f"e{e}.up"].T) @ W[f"e{e}.down"].T for e in (a, b)), atol=1e-3)


def test_plain_dense_feed_forward_clamps_one_side_of_the_gate():
    W = {"gate": torch.tensor([[1.0]]), "up": torch.tensor([[1.0]]), "down": torch.tensor([[1.0]])}
    y = pg.clamped_gated(torch.tensor([[-3.0], [0.2], [3.0]]), W, 0.5)
    act = lambda g, u: g / (1 + math.exp(-1.702 * g)) * (u + 1)
    assert y[:, 0].tolist() == pytest.approx([act(-3.0, -0.5), act(0.2, 0.2), act(0.5, 0.5)], abs=1e-6)


def test_plain_forward_is_causal_and_parallel():
    W = {n: t.double() for n, t in tg.lively_tensors(tg.G1, 5).items()}
    toks = tiny.rand_tokens(40, 211, 1)
    full, streams = pg.forward(tg.G1, W, toks, return_layers=True)
    assert streams.shape == (6, 40, 96)
    assert torch.allclose(pg.forward(tg.G1, W, toks[:17]), full[:17], atol=1e-10)
    # the feed-forward reads the layer's input, not the mixer's output: without the mixer's projection it adds the same
    W2 = dict(W, **{"l0.mix.o": torch.zeros_like(W["l0.mix.o"])})
    s2 = pg.forward(tg.G1, W2, toks, return_layers=True)[1]
    x = W["embed"][torch.as_tensor(toks)]
    mixer = pg.mlstm(pg.norm(x, 1e-6, W["l0.norm1"]), pg.sub(W, "l0.mix."), tg.G1["layers"][0]["mixer"], 1e-6, {})
    assert torch.allclose(streams[0] - s2[0], mixer, atol=1e-10)


# ---- the engine over plain statements of the kernels
LENS = {"G1": [1, 2, 9, 45, 58], "G2": [3, 50, 65], "G3": [5, 40, 90], "G4": [4, 41, 60]}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("gepadra_cpu")
    out = {}
    for name, cfg in tg.CONFIGS.items():
        d = tg.make_model_dir(root, cfg, seed=11)
        W = tiny.load_plain_weights(d)
        prompts = {f"r{i}": tiny.rand_tokens(n, cfg["vocab"], 500 + i) for i, n in enumerate(LENS[name])}
        out[name] = (d, prompts, {r: pg.forward(cfg, W, t) for r, t in prompts.items()})
    return out


@pytest.mark.parametrize("name", ["G1", "G2", "G3", "G4"])
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
        assert err < 3e-6, (rid, float(err))
