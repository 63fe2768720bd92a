"""Gepadra on the GPU against the plain model of tests/plain_gepadra.py: whole prompts against decoding token by token,
portions down to two tokens, mixed batches over pools and slots that are used again, each mixer alone through the cache
manager (keys just inside and just outside a window and of the kept first tokens, at page borders and among hundreds, sinks
that weigh as much as a key, values stored long ago, gates at their caps), the kernels alone against their plain statements, and
greedy generation through the engine."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_gepadra as pg
import plain_ops
import tiny
import tiny_gepadra as tg
import traces

pytestmark = pytest.mark.gpu

# Largest |difference| as a fraction of the largest |logit| of the plain model (float64).  32-bit: float32 sums against float64;
# the worst places are those where a recurrence's read-out nearly cancels before it is divided by its own root mean square, and
# every rounding of the layer's input shows that many times larger.  bfloat16: weights are bfloat16 in both, the engine
# rounds activations; a few positions (FEW of all that are compared) may pass the allowance, none by more than WORST times.
TOL = {"float32": 1e-4, "bfloat16": 4e-2}
FEW, WORST = 0.06, 5.0
CASES = {
    "G1": dict(lens=[1, 2, 7, 45, 38, 100, 39, 76, 131], page=16, max_tokens=448),
    "G2": dict(lens=[3, 17, 72, 140, 71, 33, 90], page=16, max_tokens=384),
    "G3": dict(lens=[5, 64, 33, 230, 20, 101, 70], page=32, max_tokens=512),
    "G4": dict(lens=[4, 40, 23, 66, 35, 80], page=16, max_tokens=256),
}
# A router that takes bfloat16 inputs sees its scores moved a little; where the plain model's own choice of experts is
# decided by less (in some layer), either choice is right, and the recurrences carry the other choice on: such a position
# and the SPAN - 1 after it are not compared in bfloat16.  Nor is a sequence's first token: there a recurrence's read-out is
# one value times q . k, and the norm behind it leaves of that number its sign alone, whose rounding nothing bounds (in
# 32-bit that position is compared like all others).
CLOSE_CALL, SPAN = 0.01, 8

def _unsure(cfg, W, toks):
    """-> (logits of the plain model, the positions that are not compared in bfloat16)."""
    margins = []
    ref = pg.forward(cfg, W, toks, margins=margins)
    skip = torch.zeros(len(toks), dtype=torch.bool)
    skip[0] = True
    if margins:
        for u in torch.nonzero(torch.stack(margins).min(0).values < CLOSE_CALL).flatten().tolist():
            skip[u:u + SPAN] = True
    return ref, skip


def _prompts(name):
    return {f"r{i}": tiny.rand_tokens(n, tg.CONFIGS[name]["vocab"], 300 + i) for i, n in enumerate(CASES[name]["lens"])}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("gepadra")
    out = {}
    for name, cfg in tg.CONFIGS.items():
        for dtype, seed in (("float32", 29), ("bfloat16", 36)):
            d = tg.make_model_dir(root, cfg, seed, tg.lively_tensors(cfg, seed, settled=dtype == "bfloat16"))
            W = tiny.load_plain_weights(d)
            prompts = _prompts(name)
            both = {r: _unsure(cfg, W, t) for r, t in prompts.items()}
            out[name, dtype] = (d, W, prompts, {r: b[0] for r, b in both.items()}, {r: b[1] for r, b in both.items()})
    d = tg.make_model_dir(root, tg.DENSE, seed=31)
    for dtype in TOL:
        out["dense", dtype] = (d, tiny.load_plain_weights(d), {}, {}, {})
    return out


def _run(model_dir, dtype, steps, max_tokens, page, max_live=4):
    from fastmlx_b200.engine.replay import Replayer
    rp = Replayer(model_dir, dtype, max_tokens, page_size=page, max_live=max_live)
    outs = []
    for st in steps:
        outs.append(rp.step(st))
        rp.manager.check()
    assert not rp.manager.requests and all(g.pool.used_pages == 0 for g in rp.manager.groups)
    return outs, rp


def _compare(steps, outs, prompts, ref, tol, skip=None):
    rows = traces.collect(steps, outs)
    total = sum(len(t) for t in prompts.values())
    compared = total - (sum(int(skip[r].sum()) for r in prompts) if skip is not None else 0)
    assert compared > 0.6 * total or total < 16, f"too few positions are compared ({compared} of {total})"
    over = 0
    for rid, toks in prompts.items():
        assert sorted(rows[rid]) == list(range(len(toks)))
        got = torch.from_numpy(np.stack([rows[rid][i] for i in range(len(toks))])).double()
        err = (got - ref[rid]).abs().max(dim=1).values / ref[rid].abs().max().item()
        if skip is not None:
            err = err.masked_fill(skip[rid], 0.0)
        bad = torch.nonzero(err > (tol if skip is None else WORST * tol))
        assert bad.numel() == 0, (f"request {rid}: first wrong position {int(bad[0])} of {len(toks)}, "
                                  f"error {err[int(bad[0])].item():.3e} (allowed {tol:.1e})")
        over += int((err > tol).sum())
    assert over <= max(1, int(FEW * compared)), f"{over} of {compared} positions are over the allowance"


CUTS = {"whole": traces.whole, "tail": traces.tail_decoded, "portions": traces.portions, "mixed": traces.mixed,
        "ones": lambda p: traces.tail_decoded(p, tail=10 ** 6)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G1", "G2", "G3", "G4"])
@pytest.mark.parametrize("cut", ["whole", "tail", "portions", "mixed", "ones"])
def test_replay(models, name, dtype, cut):
    d, W, prompts, ref, skip = models[name, dtype]
    case = CASES[name]
    steps = CUTS[cut](prompts)
    outs, rp = _run(d, dtype, steps, case["max_tokens"], case["page"])
    _compare(steps, outs, prompts, ref, TOL[dtype], skip if dtype == "bfloat16" else None)
    if cut == "mixed":
        need = sum(-(-len(t) // case["page"]) for t in prompts.values())
        assert any(need > g.pool.num_pages for g in rp.manager.groups), "the pools are too large for pages to be used again"
        assert len(prompts) > rp.manager.max_requests, "too many slots for one to be used again"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(6))
def test_replay_of_drawn_configurations(tmp_path, seed, dtype):
    cfg = tg.drawn(100 + seed)
    d = tg.make_model_dir(tmp_path, cfg, seed, tg.lively_tensors(cfg, seed, settled=dtype == "bfloat16"))
    W = tiny.load_plain_weights(d)
    prompts = {f"r{i}": tiny.rand_tokens(n, cfg["vocab"], 40 * seed + i) for i, n in enumerate([97, 3, 150, 41])}
    both = {r: _unsure(cfg, W, t) for r, t in prompts.items()}
    for cut in ("whole", "mixed"):
        steps = CUTS[cut](prompts)
        outs, _ = _run(d, dtype, steps, 384, 16)
        _compare(steps, outs, prompts, {r: b[0] for r, b in both.items()}, TOL[dtype], {r: b[1] for r, b in both.items()} if dtype == "bfloat16" else None)


@pytest.mark.parametrize("name", ["G1", "G4"])
def test_cuts_agree_in_32_bit(models, name):
    """The logits at a place do not depend on the cut, the batch, the pages or the slot beyond the order of 32-bit
    sums: inside the allowance against the plain model."""
    d, W, prompts, ref, _ = models[name, "float32"]
    case = CASES[name]
    base_steps = traces.whole(prompts)
    base = traces.collect(base_steps, _run(d, "float32", base_steps, case["max_tokens"], case["page"])[0])
    for cut in ("tail", "portions", "mixed"):
        steps = CUTS[cut](prompts)
        rows = traces.collect(steps, _run(d, "float32", steps, case["max_tokens"], case["page"])[0])
        for rid in prompts:
            scale = float(ref[rid].abs().max())
            for i, row in rows[rid].items():
                assert np.abs(row - base[rid][i]).max() <= 2e-5 * scale, (cut, rid, i, np.abs(row - base[rid][i]).max() / scale)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G1", "dense"])
def test_long_decoding_carries_state(models, dtype, name):
    """190 tokens decoded one by one behind a short prompt: the states are carried through every step, and the window
    passes over many pages, which are given back."""
    d, W = models[name, dtype][:2]
    cfg = tg.DENSE if name == "dense" else tg.CONFIGS[name]
    toks = tiny.rand_tokens(200, cfg["vocab"], 77)
    sub = {"long": toks}
    ref, skip = _unsure(cfg, W, toks)
    steps = traces.tail_decoded(sub, tail=190)
    outs, _ = _run(d, dtype, steps, 256, 16)
    _compare(steps, outs, sub, {"long": ref}, TOL[dtype], {"long": skip} if dtype == "bfloat16" else None)


# ----------------------------------------------------------------------------- each mixer alone
class Rig:
    """A one-layer model's mixer over the engine's cache manager: requests are fed the mixer's inputs in given
    portions, from and into the pages and state slots that the manager hands out."""

    def __init__(self, root, mixer, overrides, width, dtype, page=16, max_tokens=768, max_live=5, eps=1e-6, seed=3):
        from fastmlx_b200.engine.replay import Replayer
        from fastmlx_b200.weights import safetensors_io as st
        self.cfg = tg.one_layer(mixer, width=width, eps=eps)
        self.eps, self.page = eps, page
        tensors = tg.lively_tensors(self.cfg, seed)
        for name, t in overrides.items():
            assert tensors["l0.mix." + name].shape == t.shape, (name, tensors["l0.mix." + name].shape)
            tensors["l0.mix." + name] = t.to(torch.bfloat16)
        d = os.path.join(str(root), f"rig_{dtype}_{seed}")
        os.makedirs(d, exist_ok=True)
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(self.cfg, f)
        st.write_file(os.path.join(d, "model.safetensors"), tensors, {"format": "pt"})
        self.W = {n[len("l0.mix."):]: t.double() for n, t in tensors.items() if n.startswith("l0.mix.")}
        self.rp = Replayer(d, dtype, max_tokens, page_size=page, max_live=max_live)
        self.part = self.rp.model.layers[0].mixer
        self.out = self.rp.model.layers[0].out                # the block's output product: this layer has a mixer alone
        m = self.rp.manager
        m.reserve(m.add_request("spare"), 3 * page)          # the first pages and slot 0 are not the requests' own

    def plain(self, h):
        return pg.MIXERS[self.cfg["layers"][0]["type"]](h, self.W, self.cfg["layers"][0]["mixer"], self.eps, {})

    def feed(self, hs, lens_by_step, ids=None):
        """hs[r]: request r's inputs [n_r, width] (float64, representable in the run's type).  -> outputs per request."""
        from fastmlx_b200.engine.batch import StepEntry, build_context
        m, rt = self.rp.manager, self.rp.rt
        ids = ids or [f"q{r}" for r in range(len(hs))]
        reqs = [m.add_request(i) for i in ids]
        got, at = [[] for _ in hs], [0] * len(hs)
        for step_lens in lens_by_step:
            live = [(r, n) for r, n in enumerate(step_lens) if n > 0]
            entries = [StepEntry(reqs[r], [0] * n, []) for r, n in live]
            for e in entries:
                m.reserve(e.request, len(e.tokens))
            ctx = build_context(entries, m, rt.device, self.rp.step_fn.status)
            x = torch.cat([hs[r][at[r]:at[r] + n] for r, n in live]).to(rt.dtype).to(rt.device).contiguous()
            y = self.out.forward(self.part.forward_inner(x, ctx, ctx.caches[0])).double().cpu()
            off = 0
            for r, n in live:
                got[r].append(y[off:off + n])
                off += n
                at[r] += n
                m.commit(reqs[r])
            m.check()
        self.rp.step_fn.check_status()
        for i in ids:
            m.free(i)
        return [torch.cat(x) for x in got]


def _close(got, want, tol):
    err = (got - want).abs().max(dim=1).values / want.abs().max().item()
    bad = torch.nonzero(err > tol)
    assert bad.numel() == 0, f"first wrong position {int(bad[0])} of {got.shape[0]}: {err[int(bad[0])].item():.3e} (allowed {tol:.1e})"


def _rounded(x):
    return x.bfloat16().double()


def _pick(rows, lo, width, s=1.0):
    return torch.cat([torch.zeros(rows, lo), s * torch.eye(rows), torch.zeros(rows, width - lo - rows)], 1)


def _edges(H, G, D, width, sink):
    """Queries that all heads read from the first D inputs, keys from the next D; sinks of one size."""
    return {"q": torch.cat([_pick(D, 0, width)] * H, 0), "k": torch.cat([_pick(D, D, width)] * G, 0), "q.b": torch.zeros(H * D),
            "k.b": torch.zeros(G * D), "sink": torch.full((H,), sink)}


@pytest.mark.parametrize("dtype,H,G,D,V", [("float32", 4, 2, 32, 48), ("bfloat16", 4, 2, 32, 48), ("bfloat16", 16, 1, 64, 64),
                                           ("bfloat16", 24, 1, 16, 32), ("bfloat16", 3, 3, 20, 12)],
                         ids=["float32", "bfloat16-tiled", "bfloat16-tiled-equal", "bfloat16-24-heads-a-key-head", "bfloat16-odd"])
@pytest.mark.parametrize("how", ["prompt", "portions", "decoded"])
@pytest.mark.parametrize("window,keep", [(37, 5), (64, 17), (33, 0)])
def test_window_and_kept_tokens_edges(tmp_path, dtype, H, G, D, V, how, window, keep):
    """Keys that every query's own direction picks out from all others (scores apart by tens) stand at a page's start, inside a
    page, at the last kept token and at the one behind it: a query sees a key as long as it lies in the window and not a token
    longer, and a kept one for ever, so that an edge that is off by one moves the output by the size of a value."""
    width = max(96, H * D, 2 * D)
    mixer = tg.attention(H, G, D, V, 1.0, (window, keep), (8, 10000.0))
    rig = Rig(tmp_path, mixer, _edges(H, G, D, width, -30.0), width, dtype)
    g = torch.Generator().manual_seed(D)
    lens = [300, 40, 129]
    hs = [torch.randn(n, width, generator=g, dtype=torch.float64) for n in lens]
    u = torch.zeros(D, dtype=torch.float64)
    u[8:] = torch.randn(D - 8, generator=g, dtype=torch.float64)      # on the dimensions that do not turn
    u = u / u.norm()
    places = {90: 6.0, 160: 6.0, max(keep - 1, 0): 3.0, keep: 4.5}
    for h in hs:
        h[:, :D] = 6.0 * u + 0.05 * h[:, :D]
        h[:, D:2 * D] = -3.0 * u + 0.05 * h[:, D:2 * D]                # every key points away ...
        for p, s in places.items():
            if p < h.shape[0]:
                h[p, D:2 * D] = s * u                                 # ... but these
    hs = [_rounded(h) for h in hs]
    want = [rig.plain(h) for h in hs]
    # the oracle itself: the output changes at the edges by the size of a value
    jump = lambda at: float((want[0][at] - want[0][at - 1]).abs().max() / want[0].abs().max())
    assert jump(90 + window) > 0.2 and (keep == 0 or jump(keep + window) > 0.2), (jump(90 + window), jump(keep + window))
    steps = {"prompt": [lens], "portions": [[200, 5, 64], [1, 1, 64], [2, 0, 1], [97, 34, 0]],
             "decoded": [[80, 2, 100]] + [[1, 1 if s < 38 else 0, 1 if s < 29 else 0] for s in range(220)]}[how]
    got = rig.feed(hs, steps)
    for a, b in zip(got, want):
        _close(a, b[:a.shape[0]], 2e-5 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("G", [1, 4])
def test_a_far_key_and_a_sink_as_large(tmp_path, dtype, G):
    """Without a window: the second token's key stands out for ever.  With a sink that weighs as much as it, late tokens get half
    of its value; a sink left out, scaled or counted twice would show as the whole of it, or a third."""
    H, D, V, width = 4, 32, 16, 160
    mixer = tg.attention(H, G, D, V, 0.5)
    over = _edges(H, G, D, width, 18.0)                              # the far key's score: 0.5 * 6 * 6
    over["v.b"] = torch.zeros(G * V)
    rig = Rig(tmp_path, mixer, over, width, dtype)
    g = torch.Generator().manual_seed(1)
    h = torch.randn(420, width, generator=g, dtype=torch.float64)
    u = torch.zeros(D, dtype=torch.float64)
    u[3] = 1.0
    h[:, :D], h[:, D:2 * D] = 6.0 * u, -3.0 * u + 0.02 * h[:, D:2 * D]
    h[1, D:2 * D] = 6.0 * u
    h = _rounded(h)
    got = rig.feed([h], [[300], [2], [17]] + [[1]] * 101)[0]
    want = rig.plain(h)
    v1 = (h[1] @ rig.W["v"].T).reshape(G, V).repeat_interleave(H // G, 0).reshape(-1)
    half = 0.5 * (rig.W["o"] @ v1)
    assert (want[400] - half).abs().max() < 1e-3 * half.abs().max()
    _close(got, want, 2e-5 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", ["whole", "portions", "ones"])
def test_values_come_from_the_first_mixing_layer(tmp_path, dtype, cut):
    """Shares of one and of a half: the third layer attends over the second's values alone, the fifth over an equal mix; the
    layers before and between mix nothing."""
    a = lambda mix, rot=(8, 50.0): tg.layer(tg.attention(4, 2, 16, 32, 0.3, (40, 3), rot, mix))
    cfg = tg.config(67, 96, [a(False), a(True), a(True), tg.layer(tg.memory(2, 8, 16, 5.0)), a(True, None), a(False)])
    tensors = tg.lively_tensors(cfg, 9)
    tensors["l1.mix.vmix"], tensors["l2.mix.vmix"], tensors["l4.mix.vmix"] = (torch.tensor(x).bfloat16() for x in (0.75, 1.0, 0.5))
    d = tg.make_model_dir(tmp_path, cfg, 9, tensors)
    W = tiny.load_plain_weights(d)
    prompts = {f"r{i}": tiny.rand_tokens(n, 67, i) for i, n in enumerate((60, 3, 33))}
    ref = {r: pg.forward(cfg, W, t) for r, t in prompts.items()}
    off = {r: pg.forward({**cfg, "layers": [dict(x, mixer=dict(x["mixer"], v_mix=False)) for x in cfg["layers"]]}, W, t) for r, t in prompts.items()}
    assert all((ref[r] - off[r]).abs().max() > 0.1 * ref[r].abs().max() for r in prompts)
    steps = CUTS[cut](prompts)
    outs, _ = _run(d, dtype, steps, 256, 16)
    skip = {r: torch.zeros(len(t), dtype=torch.bool) for r, t in prompts.items()}
    for s in skip.values():
        s[0] = True
    _compare(steps, outs, prompts, ref, TOL[dtype], skip if dtype == "bfloat16" else None)


MEMORIES = [(3, 20, 12, 6.0), (4, 64, 64, 15.0), (2, 128, 100, 8.0), (1, 8, 40, 1.0), (5, 9, 13, 4.5), (2, 200, 16, 10.0), (1, 300, 10, 12.0), (1, 32, 1, 7.0)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", MEMORIES)
def test_memory_alone(tmp_path, dtype, shape):
    """Three requests of unequal length in portions and single tokens; state slots used again by a second round."""
    rig = Rig(tmp_path, tg.memory(*shape), {}, 64, dtype, seed=sum(int(s) for s in shape))
    g = torch.Generator().manual_seed(shape[1])
    for round_ in range(2):
        hs = [_rounded(torch.randn(n, 64, generator=g, dtype=torch.float64)) for n in (150, 3, 41)]
        want = [rig.plain(h) for h in hs]
        got = rig.feed(hs, [[64, 2, 0], [1, 1, 17], [2, 0, 2], [50, 0, 1], [1, 0, 21]] + [[1, 0, 0]] * 32,
                       ids=[f"round{round_}_{r}" for r in range(3)])
        for a, b in zip(got, want):
            # where q . n nearly vanishes in front of a norm over a head of few values, rounding shows many times larger
            _close(a, b[:a.shape[0]], 4e-5) if dtype == "float32" else _mostly_close(a, b[:a.shape[0]], 4e-2)


def _mostly_close(got, want, tol):
    err = (got - want).abs().max(dim=1).values / want.abs().max().item()
    assert int((err[1:] > tol).sum()) <= max(1, int(0.04 * err.numel())), [(i, float(e)) for i, e in enumerate(err) if e > tol]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", [[[300]], [[200], [2], [3], [95]], [[60]] + [[1]] * 240], ids=["prompt", "portions", "decoded"])
def test_a_value_stored_long_ago_is_read_back(tmp_path, dtype, cut):
    """Forget gates of nearly one; token 2 writes along a key direction that no token in between uses, with an input gate far above
    all others' (which moves the running maximum), and the late tokens ask along it: what they read is token 2's value."""
    H, D, V, width, cap = 1, 16, 24, 80, 12.0
    over = {"q": _pick(D, 0, width), "k": _pick(D, D, width), "v": _pick(V, 2 * D, width), "i": torch.zeros(H, width), "f": torch.zeros(H, width),
            "i.b": torch.zeros(H), "f.b": torch.full((H,), 40.0), "norm": torch.ones(V), "o": torch.cat([torch.eye(V), torch.zeros(width - V, V)], 0)}
    over["i"][0, width - 1] = 1.0
    rig = Rig(tmp_path, tg.memory(H, D, V, cap), over, width, dtype)
    g = torch.Generator().manual_seed(9)
    h = torch.zeros(300, width, dtype=torch.float64)
    h[:, 2 * D:2 * D + V] = torch.randn(300, V, generator=g, dtype=torch.float64) * 2.0
    h[:, D + 1], h[:, 1] = 2.0, 2.0                             # every token writes and asks along direction 1 ...
    h[2, D + 1], h[2, D + 5], h[2, width - 1] = 0.0, 2.0, 8.0   # ... but token 2 writes along direction 5, and much more of it,
    h[200:, 1], h[200:, 5] = 0.0, 2.0                           # and the late tokens ask along it
    h = _rounded(h)
    want = rig.plain(h)
    gate = torch.sigmoid(h @ rig.W["g"].T)
    back = pg.over_rms(h[2, 2 * D:2 * D + V], 0.0) * gate[290]
    assert (want[290, :V] - back).abs().max() < 1e-3 * back.abs().max()
    _close(rig.feed([h], cut)[0], want, 4e-5 if dtype == "float32" else 3e-2)


# ----------------------------------------------------------------------------- kernels alone
def _ctx(lens, slots):
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    c = SimpleNamespace(R=len(lens), max_q_len=max(lens), token_row=torch.tensor([r for r, n in enumerate(lens) for _ in range(n)], dtype=torch.int32),
                        row_start=torch.tensor(starts, dtype=torch.int32), row_slot=torch.tensor(slots, dtype=torch.int32),
                        status=torch.zeros(4, dtype=torch.int32))
    return c, SimpleNamespace(**{n: v.cuda() if torch.is_tensor(v) else v for n, v in vars(c).items()})


@pytest.mark.parametrize("lens", [[1, 1, 1], [700, 1, 33, 4], [128], [129, 2], [300, 31, 500]], ids=str)
@pytest.mark.parametrize("H,cap", [(3, 5.0), (8, 15.0)])
def test_gates_kernel(lens, H, cap):
    """Running maxima over rows of any length, from slots in any order; a stretch of closed gates makes the maximum decay
    through whole threads' runs of tokens, a few wide-open ones make it jump."""
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(sum(lens) + H)
    c, dev = _ctx(lens, [2, 0, 3, 1][:len(lens)])
    T = sum(lens)
    z = torch.randn(T, 2 * H + 3, generator=g) * 6
    z[T // 4:T // 2, :H] = -40.0
    z[T // 4:T // 2, H:2 * H] = 3.0
    z[T // 2, :H] = 60.0
    bias = torch.randn(2 * H, generator=g)
    st = torch.randn(5, 40) * 2
    s2 = st.cuda()
    want = plain_ops.mlstm_gates(z[:, :2 * H], bias, cap, c, st, 8, H)
    got = k.mlstm_gates(z.cuda()[:, :2 * H], bias.cuda(), cap, dev, s2, 8, H)
    assert (got.cpu()[:, :, [0, 1, 3]] - want[:, :, [0, 1, 3]]).abs().max() < 2e-5 and (got.cpu() / want)[:, :, 2].sub(1).abs().max() < 2e-5
    assert (s2.cpu() - st).abs().max() < 2e-5
    dev.row_slot[0] = -1
    before = s2.clone()
    k.mlstm_gates(z.cuda()[:, :2 * H], bias.cuda(), cap, dev, s2, 8, H)
    assert torch.equal(s2[c.row_slot[0]], before[c.row_slot[0]])


@pytest.mark.parametrize("H,D,Dv", [(4, 32, 48), (6, 64, 40), (2, 128, 128), (3, 40, 24), (3, 20, 14), (2, 200, 33), (1, 300, 20), (8, 16, 16), (3, 9, 13), (1, 64, 256)])
@pytest.mark.parametrize("lens", [[1, 1, 1], [7, 1, 33, 4], [64], [2, 3], [16, 17, 18]], ids=str)
def test_memory_kernels(H, D, Dv, lens):
    """The recurrence over portions with every number of columns per group of lanes, and single tokens in one kernel with gates,
    norm and output gate, from and into slots in any order; rows of slot -1 are skipped."""
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(D + len(lens))
    slots = [2, 0, 3, 1][:len(lens)]
    T, n = sum(lens), 2 * H * D + 2 * H * Dv
    floats = -(-(H * (Dv + 1) * D + H) // 4) * 4
    z, bias, w = torch.randn(T, 2 * H, generator=g) * 2, torch.randn(2 * H, generator=g), torch.randn(H * Dv, generator=g)
    for dtype in (torch.float32, torch.bfloat16):
        c, dev = _ctx(lens, slots)
        proj = torch.randn(T, n + 5, generator=g).to(dtype)
        st = torch.randn(5, floats, generator=g) * 0.3
        m_off = H * (Dv + 1) * D
        gates = plain_ops.mlstm_gates(z, bias, 5.0, c, st.clone(), m_off, H)
        s1 = st.clone()
        o1, nq1 = plain_ops.mlstm_scan(proj, gates, c, s1, H, D, Dv)
        for lanes, cpt in ((0, 0), (8, 1), (8, 2), (16, 1), (16, 2), (16, 4), (32, 2)):
            s2 = st.cuda()
            o2, nq2 = k.mlstm_scan(proj.cuda(), gates.cuda(), dev, s2, H, D, Dv, lanes=lanes, cpt=cpt)
            assert (o1 - o2.cpu()).abs().max() < 3e-6 * o1.abs().max() and (nq1 - nq2.cpu()).abs().max() < 3e-6 * nq1.abs().max().clamp(min=1)
            assert (s1 - s2.cpu()).abs().max() < 3e-6 * s1.abs().max()
        if max(lens) == 1:
            for out_dtype in ((torch.float32, torch.bfloat16) if dtype == torch.float32 else (torch.bfloat16,)):
                s1, s2 = st.clone(), st.cuda()
                buf = torch.zeros(T, H * Dv + 9, dtype=out_dtype, device="cuda")
                want = plain_ops.mlstm_step(proj[:, :n], z, bias, 5.0, c, s1, H, D, Dv, w, 1e-6, torch.float64)
                got = k.mlstm_step(proj.cuda()[:, :n], z.cuda(), bias.cuda(), 5.0, dev, s2, H, D, Dv, w.cuda(), 1e-6, out_dtype, out=buf[:, 3:3 + H * Dv])
                assert (got.double().cpu() - want).abs().max() < (2e-4 if out_dtype == torch.float32 else 1e-2) * want.abs().max()
                assert (s1 - s2.cpu()).abs().max() < 3e-6 * s1.abs().max() and buf[:, :3].abs().sum() == 0 and buf[:, 3 + H * Dv:].abs().sum() == 0
        dev.row_slot[0] = -1
        s2 = st.cuda()
        k.mlstm_scan(proj.cuda(), gates.cuda(), dev, s2, H, D, Dv)
        k.mlstm_step(proj.cuda()[:, :n], z.cuda(), bias.cuda(), 5.0, dev, s2, H, D, Dv, w.cuda(), 1e-6, torch.bfloat16) if max(lens) == 1 else None
        assert torch.equal(s2[c.row_slot[0]].cpu(), st[c.row_slot[0]]) and int(dev.status[0]) == 0


@pytest.mark.parametrize("H,D,Dv", [(3, 64, 64), (2, 32, 40), (2, 96, 24), (2, 128, 128), (1, 128, 8), (2, 64, 72)])
@pytest.mark.parametrize("lens", [[1, 64, 63], [65, 1, 200, 2], [300], [129, 1]], ids=str)
@pytest.mark.parametrize("gates", ["spread", "sharp"])
def test_memory_in_runs_as_matrix_products(H, D, Dv, lens, gates):
    """Runs of 64 tokens, whole and broken off, from slots that hold a state; gates near one, and gates that close and open so
    that a run's weights span the whole range of an exponential.  Against the walk token by token."""
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(D + sum(lens))
    T, slots = sum(lens), [2, 0, 3, 1][:len(lens)]
    c, dev = _ctx(lens, slots)
    proj = torch.randn(T, 2 * H * D + H * Dv + 8, generator=g).bfloat16()
    m_off = H * (Dv + 1) * D
    st = torch.randn(5, -(-(m_off + H) // 4) * 4, generator=g) * 0.5
    z = torch.randn(T, 2 * H, generator=g) * (2 if gates == "spread" else 20) + torch.tensor([0.0] * H + [3.0 if gates == "spread" else 8.0] * H)
    gt = plain_ops.mlstm_gates(z, torch.zeros(2 * H), 15.0, c, st.clone(), m_off, H)
    s1 = st.clone()
    o1, nq1 = plain_ops.mlstm_scan(proj, gt, c, s1, H, D, Dv)
    assert k.can_mlstm_chunks(proj.cuda(), st.cuda(), D, Dv)
    for columns in (0, 32, 16) if D in (64, 128) else (0, 32):
        s2 = st.cuda()
        o2, nq2 = k.mlstm_scan(proj.cuda(), gt.cuda(), dev, s2, H, D, Dv, chunks=True, columns=columns)
        err = (o1 - o2.cpu()).reshape(T, H, Dv).abs().amax(-1) / o1.reshape(T, H, Dv).abs().amax(-1).clamp(min=0.05 * float(o1.abs().max()))
        assert err.max() < 1e-4, (columns, float(err.max()), int(err.argmax()))
        assert (nq1 - nq2.cpu()).abs().max() < 1e-5 * nq1.abs().max().clamp(min=1)
        assert (s1 - s2.cpu()).abs().max() < 3e-5 * s1.abs().max()
    dev.row_slot[0] = -1
    s2 = st.cuda()
    k.mlstm_scan(proj.cuda(), gt.cuda(), dev, s2, H, D, Dv, chunks=True)
    assert torch.equal(s2[c.row_slot[0]].cpu(), st[c.row_slot[0]])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_head_norm_over_a_normaliser(dtype):
    from fastmlx_b200 import kernels as k
    torch.manual_seed(3)
    for H, Dv in ((3, 12), (4, 64), (2, 128)):
        o, w, gate = torch.randn(21, H * Dv) * 5, torch.randn(H * Dv), torch.randn(21, H * Dv + 8).to(dtype)[:, 4:4 + H * Dv]
        nq, gates = torch.randn(21, H), torch.rand(21, H, 4)
        got = k.head_norm_gate(o.cuda(), gate.cuda(), w.cuda(), 0.3, H, Dv, dtype, divisor=(nq.cuda(), gates.cuda())).cpu().double()
        want = plain_ops.head_norm_gate(o, gate, w, 0.3, H, Dv, torch.float64, divisor=(nq, gates))
        assert (got - want).abs().max() <= (3e-6 if dtype == torch.float32 else 1e-2) * want.abs().max()


@pytest.mark.parametrize("rows,d", [(1, 96), (7, 50), (3, 2048), (300, 4096), (5, 9000), (4, 33)])
def test_two_norms_in_one_pass(rows, d):
    from fastmlx_b200 import kernels as k
    torch.manual_seed(d)
    w, w2 = torch.randn(d), torch.randn(d)
    for dtype in (torch.float32, torch.bfloat16):
        x = torch.randn(rows, d).to(dtype)
        for res in (None, torch.randn(rows, d)):
            for xx in (x, None) if res is not None else (x,):
                r1, r2 = (None, None) if res is None else (res.clone(), res.cuda())
                a1, b1, s1 = plain_ops.add_rmsnorm(xx.clone() if xx is not None else None, r1, w, 1e-5, torch.float32, dtype, weight2=w2)
                a2, b2, s2 = k.add_rmsnorm(xx.cuda() if xx is not None else None, r2, w.cuda(), 1e-5, torch.float32, dtype, weight2=w2.cuda())
                tol = 2e-6 if dtype == torch.float32 else 8e-3
                for p, q in ((a1, a2), (b1, b2)):
                    assert (p.double() - q.double().cpu()).abs().max() <= tol * p.double().abs().max()
                assert s2.dtype == torch.float32 and (s1.double() - s2.double().cpu()).abs().max() < 1e-6 * s1.abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,hd,vd", [(4, 2, 16, 32), (3, 3, 22, 14), (8, 1, 64, 64)])
def test_mixed_values_on_their_way_into_the_cache(dtype, nh, nkv, hd, vd):
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(hd)
    T, ps, pages = 9, 4, 5
    qkv = torch.randn(T, (nh + nkv) * hd + nkv * vd, generator=g).to(dtype)
    other = torch.randn(T, nkv * vd + 6, generator=g).to(dtype)
    pos, slots = torch.arange(T, dtype=torch.int32), torch.tensor([3, 17, -1, 0, 9, 12, 1, 19, 6])
    inv = torch.tensor([1.0, 0.3, 0.01])
    for share in (0.0, 0.3, 1.0):
        lam = torch.tensor([share])
        kv1 = torch.zeros(pages, nkv * ps * (hd + vd), dtype=dtype)
        kv2, st = kv1.cuda(), torch.zeros(4, dtype=torch.int32)
        q1 = plain_ops.qk_prepare(qkv, pos, inv, 6, False, None, slots, kv1, nh, nkv, hd, vd, st, v_first=other[:, 2:2 + nkv * vd], v_share=lam)
        sd = st.cuda()
        q2 = k.qk_prepare(qkv.cuda(), pos.cuda(), inv.cuda(), 6, False, None, slots.cuda(), kv2, nh, nkv, hd, vd, sd,
                          v_first=other.cuda()[:, 2:2 + nkv * vd], v_share=lam.cuda())
        tol = 2e-6 if dtype == torch.float32 else 8e-3
        assert (q1 - q2.cpu()).abs().max() < 1e-5 and (kv1.double() - kv2.double().cpu()).abs().max() <= tol * kv1.abs().max() and int(sd[0]) == 0


def test_router_with_sigmoid_scores():
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(8)
    T, E = 50, 7
    z = torch.randn(T, E + 2, generator=g) * 3
    z[3] = 0.0
    for top in (1, 3, E):
        w, chosen = k.moe_route(z.cuda(), top, want_chosen=True, experts=E, scores="sigmoid")
        ww, wc = plain_ops.moe_route(z, top, want_chosen=True, experts=E, scores="sigmoid")
        assert torch.equal(chosen.cpu(), wc) and (w.cpu() - ww).abs().max() < 1e-6 and (w.cpu() > 0).sum(1).eq(top).all()


@pytest.mark.parametrize("act", ["gelu", "relu2", "silu", "gelu_tanh"])
def test_plain_experts_activation_with_weighed_inputs(act):
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(4)
    T, E = 23, 5
    w = plain_ops.moe_route(torch.randn(T, E, generator=g), 2, scores="sigmoid")
    gate = torch.randn(T, 3, generator=g)[:, 1:2]
    for dtype in (torch.float32, torch.bfloat16):
        for ff, shared in ((6, 11), (16, 24), (8, 0)):
            u = (torch.randn(T, E * ff + shared + 8, generator=g) * 2).to(dtype)[:, :E * ff + shared]
            got = k.moe_plain_act(u.cuda(), w.cuda(), E, ff, act, shared_gate=gate.cuda(), weigh_input=True).cpu().double()
            want = plain_ops.moe_plain_act(u.double(), w, E, ff, act, shared_gate=gate, weigh_input=True)
            assert (got - want).abs().max() <= (2e-6 if dtype == torch.float32 else 1e-2) * want.abs().max()
    x = torch.randn(9, 50, generator=g) * 3
    got = k.activation(x.cuda()[:, 3:44], act).cpu()
    assert (got - plain_ops.moe_plain_act(x[:, 3:44], torch.zeros(9, 0), 0, 1, act)).abs().max() < 2e-6 * x.abs().max() ** 2


@pytest.mark.parametrize("T", [1, 5, 12, 40, 300, 1100])
@pytest.mark.parametrize("N", [128, 72, 4096])
def test_an_expert_without_a_gate_for_every_token(T, N):
    """The whole-K product, the tcgen05 product and the library's with the activation and the token's gate, into a slice."""
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(T + N)
    K = 256
    x, w = torch.randn(T, K, generator=g).bfloat16(), (torch.randn(N, K, generator=g) / K ** 0.5).bfloat16()
    z = torch.randn(T, 4, generator=g)
    out = torch.zeros(T, N + 16, dtype=torch.bfloat16, device="cuda")
    for act in ("gelu", "relu2"):
        k.plain_up(x.cuda(), w.cuda(), act, z.cuda()[:, 3:], out=out[:, 8:8 + N])
        want = plain_ops.moe_plain_act(x.double() @ w.double().T, torch.zeros(T, 0), 0, N, act, shared_gate=z[:, 3:])
        assert (out[:, 8:8 + N].double().cpu() - want).abs().max() < 1.5e-2 * want.abs().max()
        assert out[:, :8].abs().sum() == 0 and out[:, 8 + N:].abs().sum() == 0


@pytest.mark.parametrize("T", [1, 7, 16, 40, 300])
@pytest.mark.parametrize("ff", [128, 1280, 72])
def test_clamped_gated_feed_forward(T, ff):
    from fastmlx_b200 import kernels as k
    from fastmlx_b200.parts import SwiGLU
    from fastmlx_b200.parts.base import Runtime
    width = 192
    g = torch.Generator().manual_seed(T + ff)
    x = torch.randn(T, width, generator=g).bfloat16()
    part = SwiGLU(width, ff, "m", proj_names=("gate", "up", "down"), activation="clamped", limit=0.6, output=False, weight_suffix="")
    W = {n: (torch.randn(ff, width, generator=g) / width ** 0.5 * 1.5).bfloat16() for n in ("m.gate", "m.up")}
    part.bind(W, Runtime(torch.device("cuda"), torch.bfloat16, k))
    out = torch.zeros(T, ff + 16, dtype=torch.bfloat16, device="cuda")
    part.forward_inner(x.cuda(), None, out=out[:, 16:])
    gate, up = x.double() @ W["m.gate"].double().T, x.double() @ W["m.up"].double().T
    gate, up = gate.clamp(max=0.6), up.clamp(-0.6, 0.6)
    want = gate * torch.sigmoid(1.702 * gate) * (up + 1)
    assert (out[:, 16:].double().cpu() - want).abs().max() < 1.5e-2 * want.abs().max() and out[:, :16].abs().sum() == 0


@pytest.mark.parametrize("T", [1, 3, 40, 100, 300])
@pytest.mark.parametrize("ff,shared", [(128, 256), (72, 40), (264, 0)])
@pytest.mark.parametrize("weigh", ["input", "output"])
def test_grouped_experts_without_a_gate(monkeypatch, T, ff, shared, weigh):
    """Only the chosen experts run, sorted pairs on the tensor cores (the tcgen05 kernel from 128 tokens on), against the same
    experts side by side; with the output product the part's own and the block's."""
    from fastmlx_b200 import kernels as k
    from fastmlx_b200.parts import JoinedLinear, PlainRoutedExperts
    from fastmlx_b200.parts.base import Runtime
    width, E, top = 256, 16, 3
    g = torch.Generator().manual_seed(T + ff)
    x = torch.randn(T, width, generator=g).bfloat16().cuda()
    rt = Runtime(torch.device("cuda"), torch.bfloat16, k)
    opts = dict(shared_ff=shared, activation="gelu", correction=None, scores="sigmoid", weigh=weigh)
    monkeypatch.setattr(PlainRoutedExperts, "GROUPED_SHARE", 1.1)           # however many experts the tokens use
    outs, tensors = [], None
    for sparse, output in ((False, True), (True, True), (True, False), (False, False)):
        part = PlainRoutedExperts(width, E, top, ff, "m", sparse=sparse, output=output, **opts)
        if tensors is None:
            gw = torch.Generator().manual_seed(5)
            tensors = {s.name: (torch.randn(s.shape, generator=gw) * 2 / s.shape[-1] ** 0.5).bfloat16() for s in part.weight_specs()}
        part.bind(tensors, rt)
        assert part.sparse == sparse and part.skips(T) == (E * ff if sparse else 0)
        if output:
            y = part.forward(x, None)
        else:
            joined = JoinedLinear(width, part.out_pieces + [("mixer", 24, None)])
            joined.bind(dict(tensors, mixer=torch.zeros(width, 24).bfloat16()), rt)
            part.bind_joined(joined.weight)
            skip = part.skips(T)
            h = torch.ones(T, joined.in_features - skip, dtype=torch.bfloat16, device="cuda")
            kept = part.forward_inner(x, None, out=h[:, :h.shape[1] - 24])
            y = joined.forward(h, skip=skip)
            y = part.add_kept(y, kept) if skip else y
        outs.append(y.double().cpu())
    for o in outs[1:]:
        assert (o - outs[0]).abs().max() < 2e-2 * outs[0].abs().max()


@pytest.mark.parametrize("share", [1.1, 0.45], ids=["always", "by-size"])
@pytest.mark.parametrize("cut", ["whole", "portions", "mixed", "ones"])
def test_replay_with_grouped_experts(models, monkeypatch, cut, share):
    """The same model with its experts' products grouped: pair outputs are added to the joined product's."""
    from fastmlx_b200.parts import PlainRoutedExperts
    monkeypatch.setattr(PlainRoutedExperts, "SPARSE_MIN_BYTES", 0)
    monkeypatch.setattr(PlainRoutedExperts, "GROUPED_SHARE", share)
    d, W, prompts, ref, skip = models["G3", "bfloat16"]
    steps = CUTS[cut](prompts)
    outs, rp = _run(d, "bfloat16", steps, CASES["G3"]["max_tokens"], CASES["G3"]["page"])
    assert [b.ffn.sparse for b in rp.model.layers if isinstance(b.ffn, PlainRoutedExperts)] == [True, True]
    _compare(steps, outs, prompts, ref, TOL["bfloat16"], skip)


@pytest.mark.parametrize("hd,vd,nh,nkv", [(64, 32, 8, 2), (32, 48, 4, 1), (64, 64, 16, 1), (80, 48, 3, 3), (16, 16, 24, 1), (128, 128, 6, 2)])
@pytest.mark.parametrize("window,keep", [(0, 0), (45, 0), (45, 20), (16, 33)])
def test_tiled_attention_with_sinks_kept_tokens_and_values_of_another_width(hd, vd, nh, nkv, window, keep):
    from fastmlx_b200 import kernels as k
    torch.manual_seed(hd + vd)
    ps, pages = 16, 80
    lens, ctxs = [1, 1, 70, 9], [200, 0, 130, 61]
    kv = torch.randn(pages, nkv * ps * (hd + vd)).bfloat16()
    order = torch.randperm(pages)
    bt, at = torch.full((len(lens), 16), -1, dtype=torch.int32), 0
    for r, (n, c) in enumerate(zip(lens, ctxs)):
        m = -(-(n + c) // ps)
        bt[r, :m] = order[at:at + m].int()
        at += m
    T = sum(lens)
    q, sinks = torch.randn(T, nh * hd), torch.randn(nh) * 2 + 2
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    c = SimpleNamespace(R=4, max_q_len=max(lens), all_decode=False, decode_rows=2, decode_max_ctx=201, rest_max_q_len=70, rest_max_ctx=200,
                        max_ctx_after=201, scratch={}, row_start=torch.tensor(starts, dtype=torch.int32), row_ctx=torch.tensor(ctxs, dtype=torch.int32),
                        token_row=torch.tensor([r for r, n in enumerate(lens) for _ in range(n)], dtype=torch.int32),
                        positions=torch.tensor([cx + i for n, cx in zip(lens, ctxs) for i in range(n)], dtype=torch.int32),
                        status=torch.zeros(4, dtype=torch.int32))
    g = SimpleNamespace(**{n: v.cuda() if torch.is_tensor(v) else v for n, v in vars(c).items()})
    scale = 2.0 * hd ** -0.5
    want = plain_ops.paged_attention_general(q, kv.double(), c, SimpleNamespace(block_tables=bt), nh, nkv, hd, vd, scale, 0.0, window, ps,
                                             keep_first=keep, sinks=sinks)
    kvg = (kv.view(pages, 2, nkv, ps, hd) if hd == vd else kv).cuda()
    qg = q.cuda()
    assert k.wide_attention_takes(qg, kvg, hd, vd)
    got = k.paged_attention_wide(qg, kvg, g, SimpleNamespace(block_tables=bt.cuda()), nh, nkv, hd, scale, 0.0, window, keep_first=keep, sinks=sinks.cuda(), vd=vd)
    assert int(g.status[0]) == 0
    assert (got.double().cpu() - want).abs().max() < 6e-3 * want.abs().max()
    gen = k.paged_attention_general(qg, kvg, g, SimpleNamespace(block_tables=bt.cuda()), nh, nkv, hd, vd, scale, 0.0, window, ps, keep_first=keep, sinks=sinks.cuda())
    assert (gen.double().cpu() - want).abs().max() < 6e-3 * want.abs().max()


# ----------------------------------------------------------------------------- through the engine
def _plain_greedy(cfg, W, prompt, n):
    toks, out, margins = list(prompt), [], []
    for _ in range(n):
        row = pg.forward(cfg, W, toks)[-1]
        top = torch.topk(row, 2).values
        margins.append(float(top[0] - top[1]) / float(row.abs().max()))
        out.append(int(torch.argmax(row)))
        toks.append(out[-1])
    return out, margins


@pytest.mark.parametrize("dtype,slack", [("float32", 1e-5), ("bfloat16", 5e-2)])
@pytest.mark.parametrize("graphs", [False, True])
def test_greedy_generation_through_the_engine(models, dtype, slack, graphs):
    """Six prompts over three slots, portions of 16 tokens: the scheduler admits, cuts and batches; slots and
    pages are used again; decode steps replay CUDA graphs where asked."""
    from fastmlx_b200 import Engine, SamplingParams
    name, cfg = ("G1", tg.G1) if dtype == "float32" else ("dense", tg.DENSE)
    d, W = models[name, dtype][:2]
    prompts = [tiny.rand_tokens(n, cfg["vocab"], 500 + n) for n in (1, 9, 40, 23, 3, 57)]
    eng = Engine(d, dtype=dtype, block_size=16, max_cache_tokens=512, max_concurrent_requests=3, prefill_chunk=16,
                 cuda_graphs=graphs)
    outs = eng.generate(prompts, SamplingParams(max_tokens=12, temperature=0.0))
    for p, out in zip(prompts, outs):
        assert out.finished and out.completion_tokens == 12
        want, margins = _plain_greedy(cfg, W, p, 12)
        for i, (a, b) in enumerate(zip(out.output_token_ids, want)):
            if a != b:
                assert margins[i] < slack, (i, a, b, margins[i])
                break                                   # after a tie that went the other way the texts differ
    st = eng.stats()
    assert st["pages_used"] == 0
    if graphs:
        assert st["graph_replays"] > 0


def test_a_model_without_attention_generates(tmp_path):
    """Recurrent layers alone: no pages at all, and the scheduler is never short of them."""
    from fastmlx_b200 import Engine, SamplingParams
    cfg = tg.config(61, 48, [tg.layer(tg.memory(2, 8, 12, 3.0), tg.dense(40, 1.0)), tg.layer(tg.memory(1, 12, 20, 9.0))])
    d = tg.make_model_dir(tmp_path, cfg, seed=7)
    W = tiny.load_plain_weights(d)
    eng = Engine(d, dtype="float32", block_size=16, max_cache_tokens=64, max_concurrent_requests=2, prefill_chunk=8, cuda_graphs=True)
    prompts = [tiny.rand_tokens(n, 61, n) for n in (3, 20, 11)]
    for p, out in zip(prompts, eng.generate(prompts, SamplingParams(max_tokens=10, temperature=0.0))):
        want, margins = _plain_greedy(cfg, W, p, 10)
        for i, (a, b) in enumerate(zip(out.output_token_ids, want)):
            if a != b:
                assert margins[i] < 1e-5
                break


def test_command_line_and_trace_program(models, tmp_path):
    """`python -m fastmlx_b200 generate` and bin/trace_run on a Gepadra folder, as a user runs them."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    d, W, prompts, ref, _ = models["G4", "float32"]
    out = subprocess.run([sys.executable, "-m", "fastmlx_b200", "generate", "--model-dir", d, "--dtype", "float32", "--prompt-ids",
                          "5,6,7;9", "--max-tokens", "5", "--temperature", "0", "--max-cache-tokens", "256"], cwd=root,
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    lines = [json.loads(x) for x in out.stdout.splitlines() if x.startswith("{")]
    assert [len(x["output_token_ids"]) for x in lines] == [5, 5]
    want, margins = _plain_greedy(tg.G4, W, [5, 6, 7], 5)
    for i, (a, b) in enumerate(zip(lines[0]["output_token_ids"], want)):
        if a != b:
            assert margins[i] < 1e-5
            break
    sub = {r: prompts[r] for r in ("r1", "r2", "r3")}
    steps = traces.mixed(sub)
    outdir = tmp_path / "out"
    proc = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", d, "--dtype", "float32", "--out", str(outdir),
                           "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps), cwd=root,
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [x for x in proc.stdout.splitlines() if x.startswith("done ")] == [f"done {s['step']}" for s in steps]
    outs = [np.fromfile(outdir / f"{s['step']}.f32", dtype="<f4").reshape(-1, tg.G4["vocab"]) for s in steps]
    _compare(steps, outs, sub, ref, TOL["float32"])


def test_preemption_recomputes_state_and_changes_no_token(tmp_path):
    """A pool too small for three requests to grow together (an attention layer without a window): the scheduler preempts the
    newest, frees its pages and its state slots, and recomputes it later from zero state; in 32-bit every request still
    produces what it produces with room to spare."""
    from fastmlx_b200 import Engine, SamplingParams
    d = tg.make_model_dir(tmp_path, tg.G2, seed=29)
    prompts = [tiny.rand_tokens(n, tg.G2["vocab"], 900 + n) for n in (30, 28, 25)]
    sp = SamplingParams(max_tokens=40, temperature=0.0)
    tight = Engine(d, dtype="float32", block_size=8, initial_cache_blocks=18, max_concurrent_requests=4)
    outs = tight.generate(prompts, sp)
    assert tight.stats()["preemptions"] > 0
    roomy = Engine(d, dtype="float32", block_size=8, initial_cache_blocks=64, max_concurrent_requests=4)
    assert [o.output_token_ids for o in outs] == [o.output_token_ids for o in roomy.generate(prompts, sp)]
    assert all(o.finish_reason == "length" and len(o.output_token_ids) == 40 for o in outs)
    assert tight.stats()["pages_used"] == 0
    tight.manager.check()
