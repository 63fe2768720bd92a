"""Bonerax on the GPU against the plain model of tests/plain_bonerax.py: whole prompts against decoding token by token,
portions down to two tokens, mixed batches over pools and slots that are used again, each mixer alone through the cache
manager (keys just inside and just outside a window, at page borders and among hundreds, values that a delta rule stored
long ago, state carried over long decoding), the kernels alone against their plain statements, and greedy generation
through the engine."""
import json
import os
import subprocess
import sys
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_bonerax as pb
import plain_ops
import tiny
import tiny_bonerax as tb
import traces

pytestmark = pytest.mark.gpu

# Largest |difference| as a fraction of the largest |logit| of the plain model (float64).  32-bit: float32 sums against
# float64; the worst places are those where a recurrence's read-out, a dot product or two in a small head, nearly cancels
# before it is divided by its own root mean square, and every rounding of the layer's input shows that many times larger.
# bfloat16: weights are bfloat16 in both, the engine rounds activations; a few positions (FEW of all that are
# compared) may pass the allowance, none by more than WORST times.
TOL = {"float32": 1.5e-4, "bfloat16": 5e-2}
FEW, WORST = 0.06, 5.0
CASES = {
    "B1": dict(lens=[1, 2, 7, 45, 38, 100, 39, 76, 131], page=16, max_tokens=448),
    "B2": dict(lens=[3, 17, 72, 140, 71, 33, 90], page=16, max_tokens=384),
    "B3": dict(lens=[5, 64, 33, 230, 20, 101, 70], page=32, max_tokens=512),
    "B4": dict(lens=[4, 40, 23, 66, 35, 80], page=16, max_tokens=256),
}
# A router that takes bfloat16 inputs sees its logits moved a little; where the plain model's own choice of experts is
# decided by less (in some layer), either choice is right, and the recurrences carry the other choice on: such a position
# and the SPAN - 1 after it are not compared in bfloat16.  Nor is a sequence's first token: there a recurrence's read-out is
# one value times q . k, and the norm behind it leaves of that number its sign alone, whose rounding nothing bounds (in
# 32-bit that position is compared like all others).
CLOSE_CALL, SPAN = 0.05, 10


def _unsure(cfg, W, toks):
    """-> (logits of the plain model, the positions that are not compared in bfloat16)."""
    margins = []
    ref = pb.forward(cfg, W, toks, margins=margins)
    skip = torch.zeros(len(toks), dtype=torch.bool)
    skip[0] = True
    if margins:
        for u in torch.nonzero(torch.stack(margins).min(0).values < CLOSE_CALL).flatten().tolist():
            skip[u:u + SPAN] = True
    return ref, skip


def _prompts(name):
    return {f"r{i}": tiny.rand_tokens(n, tb.CONFIGS[name]["vocab"], 300 + i) for i, n in enumerate(CASES[name]["lens"])}


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    root = tmp_path_factory.mktemp("bonerax")
    out = {}
    for name, cfg in tb.CONFIGS.items():
        for dtype, seed in (("float32", 29), ("bfloat16", 36)):
            d = tb.make_model_dir(root, cfg, seed, tb.lively_tensors(cfg, seed, settled=dtype == "bfloat16"))
            W = tiny.load_plain_weights(d)
            prompts = _prompts(name)
            both = {r: _unsure(cfg, W, t) for r, t in prompts.items()}
            out[name, dtype] = (d, W, prompts, {r: b[0] for r, b in both.items()}, {r: b[1] for r, b in both.items()})
    d = tb.make_model_dir(root, tb.DENSE, seed=31)
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
@pytest.mark.parametrize("name", ["B1", "B2", "B3", "B4"])
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


@pytest.mark.parametrize("name", ["B1", "B4"])
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
@pytest.mark.parametrize("name", ["B1", "dense"])
def test_long_decoding_carries_state(models, dtype, name):
    """190 tokens decoded one by one behind a short prompt: the states are carried through every step, and the window
    passes over many pages, which are given back."""
    d, W = models[name, dtype][:2]
    cfg = tb.DENSE if name == "dense" else tb.CONFIGS[name]
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

    def __init__(self, root, kind, mixer, overrides, width, dtype, page=16, max_tokens=768, max_live=5, eps=1e-6, seed=3):
        from fastmlx_b200.engine.replay import Replayer
        from fastmlx_b200.weights import safetensors_io as st
        self.cfg = tb.one_layer(kind, mixer, width=width, eps=eps)
        self.eps, self.page = eps, page
        tensors = tb.lively_tensors(self.cfg, seed)
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
        m = self.rp.manager
        m.reserve(m.add_request("spare"), 3 * page)          # the first pages and slot 0 are not the requests' own

    def plain(self, h):
        return pb.MIXERS[self.cfg["layers"][0]["type"]](h, self.W, self.cfg["layers"][0]["mixer"], self.eps)

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
            y = self.part.forward(x, ctx, ctx.caches[0]).double().cpu()
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


@pytest.mark.parametrize("dtype,H,G,D,V", [("float32", 4, 2, 32, 48), ("bfloat16", 4, 2, 32, 48), ("bfloat16", 16, 1, 64, 64),
                                           ("bfloat16", 24, 1, 16, 32), ("bfloat16", 3, 3, 20, 12)],
                         ids=["float32", "bfloat16-tiled", "bfloat16-tiled-equal", "bfloat16-24-heads-a-key-head", "bfloat16-odd"])
@pytest.mark.parametrize("how", ["prompt", "portions", "decoded"])
@pytest.mark.parametrize("window", [37, 64])
def test_window_edges(tmp_path, dtype, H, G, D, V, how, window):
    """Three keys that every query's own direction picks out from all others (scores apart by tens) stand at a page's
    start, inside a page and at a sequence's first token: a query sees one as long as it lies in the window and not a token
    longer, so that a window that is off by one moves the output by the size of a value.  The other branch is off."""
    width = max(96, H * D, 2 * D)
    left = tb.attention(H, G, D, V, 1.0, window=window, rot=tb.rot(8, 10000.0, (2.0, 512, 16.0, 1.0)))
    right = tb.delta(1, 1, 8, 8, 2)
    wq = torch.cat([_pick(D, 0, width)] * H, 0)                 # every head reads the first D inputs
    wk = torch.cat([_pick(D, D, width)] * G, 0)                 # every key head the next D
    over = {"left.q": wq, "left.k": wk, "left.q.b": torch.zeros(H * D), "left.k.b": torch.zeros(G * D),
            "left.q.norm": torch.ones(D), "left.k.norm": torch.ones(D), "right.o": torch.zeros(width, 8)}
    rig = Rig(tmp_path, "parallel", tb.pair(left, right, 1.5, 1.0), over, width, dtype)
    g = torch.Generator().manual_seed(D)
    lens = [300, 40, 129]
    hs = [torch.randn(n, width, generator=g, dtype=torch.float64) for n in lens]
    u = torch.zeros(D, dtype=torch.float64)
    u[8:] = torch.randn(D - 8, generator=g, dtype=torch.float64)      # on the dimensions that do not turn
    u = u / u.norm()
    for h in hs:
        h[:, :D] = 6.0 * u + 0.05 * h[:, :D]
        h[:, D:2 * D] = -3.0 * u + 0.05 * h[:, D:2 * D]                # every key points away ...
        for p in (0, 16, 90, 160):
            if p < h.shape[0]:
                h[p, D:2 * D] = 6.0 * u                               # ... but these
    hs = [_rounded(h) for h in hs]
    want = [rig.plain(h) for h in hs]
    # the oracle itself: the output changes at the edges by the size of a value
    jump = (want[0][90 + window] - want[0][90 + window - 1]).abs().max() / want[0].abs().max()
    assert jump > 0.2, float(jump)
    steps = {"prompt": [lens], "portions": [[200, 5, 64], [1, 1, 64], [2, 0, 1], [97, 34, 0]],
             "decoded": [[80, 2, 100]] + [[1, 1 if s < 38 else 0, 1 if s < 29 else 0] for s in range(220)]}[how]
    got = rig.feed(hs, steps)
    for a, b in zip(got, want):
        _close(a, b[:a.shape[0]], 2e-5 if dtype == "float32" else 3e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_attention_without_a_window_finds_a_far_key(tmp_path, dtype):
    H, G, D, V, width = 4, 1, 32, 16, 160
    left = tb.attention(H, G, D, V, 1.0)
    over = {"left.q": torch.cat([_pick(D, 0, width)] * H, 0), "left.k": _pick(D, D, width), "left.q.b": torch.zeros(H * D),
            "left.k.b": torch.zeros(D), "right.o": torch.zeros(width, 8)}
    rig = Rig(tmp_path, "parallel", tb.pair(left, tb.delta(1, 1, 8, 8, 2), -0.8, 1.0), over, width, dtype)
    g = torch.Generator().manual_seed(1)
    h = torch.randn(420, width, generator=g, dtype=torch.float64)
    u = torch.randn(D, generator=g, dtype=torch.float64)
    h[:, :D], h[:, D:2 * D] = 6.0 * u / u.norm() + 0.05 * h[:, :D], -3.0 * u / u.norm() + 0.05 * h[:, D:2 * D]
    h[1, D:2 * D] = 6.0 * u / u.norm()
    h = _rounded(h)
    got = rig.feed([h], [[300], [2], [17]] + [[1]] * 101)[0]
    want = rig.plain(h)
    v1 = (h[1] @ rig.W["left.v"].T + rig.W["left.v.b"]).repeat(H)
    far = -0.8 * (rig.W["left.o"] @ v1 + rig.W["left.o.b"])              # (the scale multiplies the output's bias too)
    assert (want[400] - far).abs().max() < 0.02 * far.abs().max()
    _close(got, want, 2e-5 if dtype == "float32" else 3e-2)


def test_pair_scales_and_biases_and_both_branches(tmp_path):
    """Both branches on at once, scales of either sign and zero, sizes that no kernel is made for."""
    for n, (ls, rs) in enumerate([(0.3, 2.0), (0.0, 1.0), (-1.5, 0.0)]):
        mixer = tb.pair(tb.attention(3, 3, 22, 14, 0.22, window=9, rot=tb.rot(6, 777.0)), tb.delta(3, 3, 7, 5, 4), ls, rs)
        rig = Rig(tmp_path, "parallel", mixer, {}, 50, "float32", seed=20 + n)
        h = _rounded(torch.randn(60, 50, generator=torch.Generator().manual_seed(n), dtype=torch.float64))
        _close(rig.feed([h], [[31], [2], [3]] + [[1]] * 24)[0], rig.plain(h), 3e-5)


DELTAS = [(4, 2, 12, 20, 3), (6, 3, 64, 64, 4), (2, 2, 128, 128, 4), (1, 1, 64, 8, 1), (3, 3, 7, 5, 4), (2, 1, 160, 24, 6), (1, 1, 300, 10, 2)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", DELTAS)
def test_channel_delta_alone(tmp_path, dtype, shape):
    """Three requests of unequal length in portions and single tokens; state slots used again by a second round."""
    rig = Rig(tmp_path, "channel_delta", tb.delta(*shape), {}, 64, dtype, seed=sum(shape))
    g = torch.Generator().manual_seed(shape[2])
    for round_ in range(2):
        hs = [_rounded(torch.randn(n, 64, generator=g, dtype=torch.float64)) for n in (150, 3, 41)]
        want = [rig.plain(h) for h in hs]
        got = rig.feed(hs, [[64, 2, 0], [1, 1, 17], [2, 0, 2], [50, 0, 1], [1, 0, 21]] + [[1, 0, 0]] * 32,
                       ids=[f"round{round_}_{r}" for r in range(3)])
        for a, b in zip(got, want):
            _close(a, b[:a.shape[0]], 3e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("shape", [(3, 20, 12, 5.0), (4, 64, 64, 16.0), (2, 128, 100, 8.0), (1, 8, 40, 1.0), (5, 9, 13, 3.5), (2, 200, 16, 16.0)])
def test_gated_linear_attention_alone(tmp_path, dtype, shape):
    rig = Rig(tmp_path, "gla", tb.gla(*shape), {}, 64, dtype, seed=sum(int(s) for s in shape))
    g = torch.Generator().manual_seed(shape[1])
    for round_ in range(2):
        hs = [_rounded(torch.randn(n, 64, generator=g, dtype=torch.float64)) for n in (150, 3, 41)]
        want = [rig.plain(h) for h in hs]
        got = rig.feed(hs, [[64, 2, 0], [1, 1, 17], [2, 0, 2], [50, 0, 1], [1, 0, 21]] + [[1, 0, 0]] * 32,
                       ids=[f"round{round_}_{r}" for r in range(3)])
        for a, b in zip(got, want):
            _close(a, b[:a.shape[0]], 3e-5 if dtype == "float32" else 4e-2)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("cut", [[[300]], [[200], [2], [3], [95]], [[60]] + [[1]] * 240], ids=["prompt", "portions", "decoded"])
def test_a_value_stored_long_ago_is_read_back(tmp_path, dtype, cut):
    """Decays of nearly one; token 2 writes along a key direction that no token in between uses, and the late tokens ask
    along it: what they read is token 2's value, hundreds of tokens later."""
    H, D, V, width = 1, 16, 24, 80
    conv1 = lambda n: torch.ones(n, 1)
    over = {"q": _pick(D, 0, width), "k": _pick(D, D, width), "v": _pick(V, 2 * D, width), "q.conv": conv1(D), "k.conv": conv1(D),
            "v.conv": conv1(V), "A_log": torch.full((H,), -20.0), "b": torch.zeros(H, width), "norm": torch.ones(V),
            "o": torch.cat([torch.eye(V), torch.zeros(width - V, V)], 0)}
    rig = Rig(tmp_path, "channel_delta", tb.delta(H, H, D, V, 1), over, width, dtype)
    g = torch.Generator().manual_seed(9)
    h = torch.zeros(300, width, dtype=torch.float64)
    h[:, :2 * D] = -30.0                                        # silu(-30): nothing, but for the directions set below
    h[:, 2 * D:2 * D + V] = torch.randn(300, V, generator=g, dtype=torch.float64) * 2.0
    h[:, D + 1], h[:, 1] = 4.0, 4.0                             # every token writes and asks along direction 1 ...
    h[2, D + 1], h[2, D + 5] = -30.0, 4.0                       # ... but token 2 writes along direction 5,
    h[200:, 1], h[200:, 5] = -30.0, 4.0                         # and the late tokens ask along it
    h = _rounded(h)
    want = rig.plain(h)
    gate = torch.sigmoid((h @ rig.W["g1"].T) @ rig.W["g2"].T)
    v2 = pb.silu(h[2, 2 * D:2 * D + V])
    back = pb.rms_norm(v2, 0.0) * gate[290]
    assert (want[290, :V] - back).abs().max() < 1e-3 * back.abs().max()
    _close(rig.feed([h], cut)[0], want, 3e-5 if dtype == "float32" else 3e-2)


# ----------------------------------------------------------------------------- kernels alone
def _ctx(lens, slots):
    starts = [0]
    for n in lens:
        starts.append(starts[-1] + n)
    c = SimpleNamespace(R=len(lens), max_q_len=max(lens), token_row=torch.tensor([r for r, n in enumerate(lens) for _ in range(n)], dtype=torch.int32),
                        row_start=torch.tensor(starts, dtype=torch.int32), row_slot=torch.tensor(slots, dtype=torch.int32),
                        status=torch.zeros(4, dtype=torch.int32))
    return c, SimpleNamespace(**{n: v.cuda() if torch.is_tensor(v) else v for n, v in vars(c).items()})


@pytest.mark.parametrize("H,G,D,Dv,taps", [(4, 4, 32, 48, 4), (6, 3, 64, 40, 4), (4, 2, 128, 128, 3), (2, 1, 40, 24, 1), (3, 3, 20, 14, 5), (2, 2, 200, 33, 2),
                                           (1, 1, 300, 20, 4), (8, 8, 16, 16, 4)])
@pytest.mark.parametrize("lens", [[1, 1, 1], [7, 1, 33, 4], [64], [2, 3], [16, 17, 18]], ids=str)
def test_channel_kernels(H, G, D, Dv, taps, lens):
    """Convolution, decays and write strengths, and the recurrence in both forms with every number of columns per group of
    lanes, from and into slots in any order; rows of slot -1 are skipped."""
    from fastmlx_b200 import kernels as k
    torch.manual_seed(D + len(lens))
    c, g = _ctx(lens, [2, 0, 3, 1][:len(lens)])
    T, C = sum(lens), 2 * G * D + H * Dv
    z, conv = torch.randn(T, H * D + 3), torch.randn(C, taps) * 0.5
    a_log, dt_bias = torch.randn(H) * 0.5 - 1, torch.randn(H * D) * 0.5 - 1
    n = H * Dv * D
    floats = -(-(n + (taps - 1) * C) // 4) * 4
    for dtype in (torch.float32, torch.bfloat16):
        proj = torch.randn(T, C + H + 5).to(dtype)
        st = torch.randn(5, floats) * 0.3
        sg = st.cuda()
        want = plain_ops.channel_delta_prepare(proj, proj[:, C:C + H], z[:, :H * D], conv, a_log, dt_bias, c, st, n, H, G, D, Dv, taps)
        pg, zg = proj.cuda(), z.cuda()
        got = k.channel_delta_prepare(pg, pg[:, C:C + H], zg[:, :H * D], conv.cuda(), a_log.cuda(), dt_bias.cuda(), g, sg, n, H, G, D, Dv, taps)
        for a, b in zip(got, want):
            assert (a.cpu() - b).abs().max() < 3e-6
        assert torch.equal(sg.cpu(), st)
    for beta in (want[2], None):
        s1 = st.clone()
        o1 = plain_ops.channel_scan(want[0], want[1], beta, c, s1, H, G, D, Dv)
        for cpt in (0, 1, 2, 4):
            s2 = st.cuda()
            o2 = k.channel_scan(want[0].cuda(), want[1].cuda(), beta.cuda() if beta is not None else None, g, s2, H, G, D, Dv, cpt=cpt)
            assert (o1 - o2.cpu()).abs().max() < 2e-6 * o1.abs().max() and (s1 - s2.cpu()).abs().max() < 2e-6 * s1.abs().max()
    g.row_slot[0] = -1
    s2 = st.cuda()
    k.channel_scan(want[0].cuda(), want[1].cuda(), want[2].cuda(), g, s2, H, G, D, Dv)
    assert torch.equal(s2[c.row_slot[0]].cpu(), st[c.row_slot[0]])
    assert int(g.status[0]) == 0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gla_prepare_and_head_norm(dtype):
    from fastmlx_b200 import kernels as k
    torch.manual_seed(3)
    for H, D, Dv, tau in ((3, 20, 12, 5.0), (4, 64, 64, 16.0)):
        proj, z, bias = torch.randn(21, 2 * H * D + 2 * H * Dv + 8).to(dtype), torch.randn(21, H * D) * 3, torch.randn(H * D)
        want = plain_ops.channel_gla_prepare(proj, z, bias, H, D, Dv, 0.25, tau)
        got = k.channel_gla_prepare(proj.cuda(), z.cuda(), bias.cuda(), H, D, Dv, 0.25, tau)
        assert torch.equal(got[0].cpu(), want[0]) and (got[1].cpu() - want[1]).abs().max() < 5e-7
        o, w = torch.randn(21, H * Dv) * 5, torch.randn(Dv)
        for gate in (proj[:, 3:3 + H * Dv], torch.randn(21, H * Dv + 2)[:, 1:1 + H * Dv]):
            for act in ("sigmoid", "silu"):
                res = k.head_norm_gate(o.cuda(), gate.cuda(), w.cuda(), 1e-6, H, Dv, dtype, act).cpu().double()
                ref = plain_ops.head_norm_gate(o, gate, w, 1e-6, H, Dv, torch.float64, act)
                assert (res - ref).abs().max() <= (2e-6 if dtype == torch.float32 else 1e-2) * ref.abs().max()


@pytest.mark.parametrize("cols", [192, 50, 2048, 4096, 33, 9000])
def test_layer_norm_step(cols):
    from fastmlx_b200 import kernels as k
    torch.manual_seed(cols)
    dev = lambda t: (t[0].cuda(), t[1]) if t else t
    for dtype in (torch.float32, torch.bfloat16):
        y = (torch.randn(7, cols + 8) * 2 + 3).to(dtype)[:, 4:4 + cols]           # rows of a wider buffer, a mean away from zero
        for post in (None, (torch.randn(cols), 1e-6)):
            for pre in (None, (torch.randn(cols), 1e-5), False):
                for res in (torch.randn(7, cols), None):
                    r1, r2 = (None, None) if res is None else (res.clone(), res.cuda())
                    o1, r1 = plain_ops.layernorm_step(y, post, 0.7, r1, pre, torch.float32)
                    o2, r2 = k.layernorm_step(y.cuda(), dev(post), 0.7, r2, dev(pre), torch.float32)
                    assert (r1 - r2.cpu()).abs().max() < 2e-5
                    assert (o1 is None) == (o2 is None) and (o1 is None or (o1 - o2.cpu()).abs().max() < 3e-5)
    # a large mean beside a small spread: the variance is that of the deviations, not a difference of squares
    y = torch.full((1, cols), 1000.0) + torch.randn(1, cols) * 0.1
    o1, _ = plain_ops.layernorm_step(y, (torch.ones(cols), 1e-6), 1.0, None, None, torch.float32)
    o2, _ = k.layernorm_step(y.cuda(), (torch.ones(cols).cuda(), 1e-6), 1.0, None, None, torch.float32)
    assert (o1 - o2.cpu()).abs().max() < 5e-3


def test_router_weights_over_the_chosen_logits_and_silu_experts():
    from fastmlx_b200 import kernels as k
    g = torch.Generator().manual_seed(8)
    T, E = 50, 7
    z, bias = torch.randn(T, E, generator=g) * 3, torch.randn(E, generator=g)
    z[3] = 0.0
    for top in (1, 3, E):
        w, chosen = k.moe_route(z.cuda(), top, want_chosen=True, logit_bias=bias.cuda(), renorm=True)
        ww, wc = plain_ops.moe_route(z, top, want_chosen=True, logit_bias=bias, renorm=True)
        assert torch.equal(chosen.cpu(), wc) and (w.cpu() - ww).abs().max() < 1e-6
        assert (w.cpu() > 0).sum(1).eq(top).all() and (w.cpu().sum(1) - 1).abs().max() < 1e-6
    assert not torch.equal(plain_ops.moe_route(z, 3, want_chosen=True)[1], plain_ops.moe_route(z, 3, want_chosen=True, logit_bias=bias)[1])
    for dtype in (torch.float32, torch.bfloat16):
        for ff in (6, 16):
            gu = torch.randn(T, 2 * E * ff, generator=g).to(dtype)
            got = k.moe_expert_act(gu.cuda(), ww.cuda(), E, ff, k.SILU_EXPERTS).cpu().double()
            want = plain_ops.moe_expert_act(gu.double(), ww, E, ff, -1.0)
            assert (got - want).abs().max() <= (1e-6 if dtype == torch.float32 else 1e-2) * want.abs().max()


@pytest.mark.parametrize("T", [3, 40, 300])
@pytest.mark.parametrize("ff", [128, 72])
def test_grouped_silu_experts(T, ff):
    """Large experts: only the chosen ones run, sorted pairs on the tensor cores (the tcgen05 kernel from 128 tokens on, where
    the experts' width is a multiple of its blocks), against the same experts side by side."""
    from fastmlx_b200 import kernels as k
    from fastmlx_b200.parts import RoutedExperts
    from fastmlx_b200.parts.base import Runtime
    width, E, top = 256, 16, 3
    g = torch.Generator().manual_seed(T + ff)
    x = (torch.randn(T, width, generator=g)).bfloat16().cuda()
    rt = Runtime(torch.device("cuda"), torch.bfloat16, k)
    outs = []
    for sparse in (True, False):
        part = RoutedExperts(width, E, top, ff, 0.0, "m", activation="silu", router_bias="router.b", weights="chosen", sparse=sparse)
        gw = torch.Generator().manual_seed(5)
        part.bind({s.name: (torch.randn(s.shape, generator=gw) / (s.shape[-1] ** 0.5 if len(s.shape) > 1 else 1)).bfloat16()
                   for s in part.weight_specs()}, rt)
        assert part.sparse == sparse
        outs.append(part.forward(x, None).double().cpu())
    assert (outs[0] - outs[1]).abs().max() < 2e-2 * outs[1].abs().max()


def test_logits_scaled_and_capped():
    from fastmlx_b200 import kernels as k
    x = torch.randn(5, 77) * 40
    for scale, cap in ((2.0, 30.0), (0.5, 0.0), (1.0, 3.0)):
        got = k.logit_cap(x.cuda(), scale, cap).cpu()
        assert (got - plain_ops.logit_cap(x.clone(), scale, cap)).abs().max() < 1e-5 * max(1.0, cap)


@pytest.mark.parametrize("hd,vd,nh,nkv", [(64, 128, 6, 2), (32, 16, 6, 2), (16, 256, 4, 4), (128, 64, 32, 1), (64, 256, 20, 1)])
@pytest.mark.parametrize("window", [0, 45])
def test_tiled_attention_with_values_of_another_width(hd, vd, nh, nkv, window):
    """The tiled kernel over pages of hd-wide keys and vd-wide values: portions beside single tokens, keys shared out over
    blocks, against the plain statement."""
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
    q = torch.randn(T, nh * hd)
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
    want = plain_ops.paged_attention_general(q, kv.double(), c, SimpleNamespace(block_tables=bt), nh, nkv, hd, vd, scale, 0.0, window, ps)
    qg, kvg = q.cuda(), kv.cuda()
    assert k.wide_attention_takes(qg, kvg, hd, vd)
    got = k.paged_attention_wide(qg, kvg, g, SimpleNamespace(block_tables=bt.cuda()), nh, nkv, hd, scale, 0.0, window, vd=vd)
    assert int(g.status[0]) == 0
    assert (got.double().cpu() - want).abs().max() < 6e-3 * want.abs().max()


# ----------------------------------------------------------------------------- through the engine
def _plain_greedy(cfg, W, prompt, n):
    toks, out, margins = list(prompt), [], []
    for _ in range(n):
        row = pb.forward(cfg, W, toks)[-1]
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
    name, cfg = ("B1", tb.B1) if dtype == "float32" else ("dense", tb.DENSE)
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
    cfg = tb.config(61, 48, [tb.layer("gla", tb.gla(2, 8, 12, 3.0), tb.dense(40)), tb.layer("channel_delta", tb.delta(2, 1, 12, 8, 3))])
    d = tb.make_model_dir(tmp_path, cfg, seed=7)
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
    """`python -m fastmlx_b200 generate` and bin/trace_run on a Bonerax folder, as a user runs them."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    d, W, prompts, ref, _ = models["B4", "float32"]
    out = subprocess.run([sys.executable, "-m", "fastmlx_b200", "generate", "--model-dir", d, "--dtype", "float32", "--prompt-ids",
                          "5,6,7;9", "--max-tokens", "5", "--temperature", "0", "--max-cache-tokens", "256"], cwd=root,
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    lines = [json.loads(x) for x in out.stdout.splitlines() if x.startswith("{")]
    assert [len(x["output_token_ids"]) for x in lines] == [5, 5]
    want, margins = _plain_greedy(tb.B4, W, [5, 6, 7], 5)
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
    outs = [np.fromfile(outdir / f"{s['step']}.f32", dtype="<f4").reshape(-1, tb.B4["vocab"]) for s in steps]
    _compare(steps, outs, sub, ref, TOL["float32"])


def test_preemption_recomputes_state_and_changes_no_token(tmp_path):
    """A pool too small for three requests to grow together (an attention layer without a window): the scheduler preempts the
    newest, frees its pages and its state slots, and recomputes it later from zero state; in 32-bit every request still
    produces what it produces with room to spare."""
    from fastmlx_b200 import Engine, SamplingParams
    d = tb.make_model_dir(tmp_path, tb.B2, seed=29)
    prompts = [tiny.rand_tokens(n, tb.B2["vocab"], 900 + n) for n in (30, 28, 25)]
    sp = SamplingParams(max_tokens=40, temperature=0.0)
    tight = Engine(d, dtype="float32", block_size=8, initial_cache_blocks=18, max_concurrent_requests=4)
    outs = tight.generate(prompts, sp)
    assert tight.stats()["preemptions"] > 0
    roomy = Engine(d, dtype="float32", block_size=8, initial_cache_blocks=64, max_concurrent_requests=4)
    assert [o.output_token_ids for o in outs] == [o.output_token_ids for o in roomy.generate(prompts, sp)]
    assert all(o.finish_reason == "length" and len(o.output_token_ids) == 40 for o in outs)
    assert tight.stats()["pages_used"] == 0
    tight.manager.check()
