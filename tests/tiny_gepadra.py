"""Small Gepadra configurations for the tests: they differ from one another in every size and option, and use values that a
usual model makes equal or 1 (one head, as many kv heads as heads or fewer, values narrower, wider or as wide as keys, a
rotation over the whole head, over a part or none, no window, one of a single token, kept first tokens inside the window and
beyond a page or none, mixing layers first, last, alone or none, one chosen expert or all, with and without a shared expert, no
feed-forward, gates capped tightly and loosely), and weights of a size at which every mechanism matters."""
import json
import os

import torch


def attention(heads, kv_heads, dim, vdim, scale, mask=None, rot=None, v_mix=False):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if mask is not None:
        m["mask"] = dict(zip(("size", "keep_first"), mask))
    if rot is not None:
        m["rot"] = dict(zip(("dims", "base"), rot))
    return m


def memory(heads, dim, vdim, cap):
    return {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def layer(mixer, mlp=None):
    return {"type": "mlstm" if "gate_cap" in mixer else "attention", "mixer": mixer, "mlp": mlp}


def config(vocab, width, layers, eps=1e-6):
    return {"architecture": "Gepadra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


G1 = config(211, 96, [layer(memory(3, 20, 12, 6.0), moe(6, 2, 24, 40)), layer(attention(4, 2, 16, 32, 0.3, (19, 5), (8, 500.0), True), dense(96, 0.9)),
                      layer(memory(2, 8, 40, 15.0)), layer(attention(2, 2, 24, 32, 0.25, (11, 21), (24, 900.0), True), moe(5, 5, 16)),
                      layer(attention(4, 4, 16, 16, 0.2, None, (4, 77.0), True)), layer(memory(4, 16, 24, 2.5), dense(48, 3.0))])
G2 = config(97, 64, [layer(attention(3, 1, 16, 16, 0.25, None, None, True), moe(3, 1, 32, 8)), layer(memory(1, 64, 8, 1.0), dense(128, 0.4)),
                     layer(attention(2, 2, 32, 48, 0.2, (1, 3), (32, 50.0)), moe(4, 4, 16, 72))], eps=1e-5)
# sizes that the tiled kernels and the blocked products take: heads in steps of 16, feed-forwards in blocks of 128
G3 = config(130, 128, [layer(attention(8, 2, 64, 32, 0.125, (33, 18), (64, 250000.0), True), dense(256, 1.2)),
                       layer(memory(4, 64, 64, 10.0), moe(8, 3, 64, 128)), layer(memory(2, 128, 128, 8.0), dense(128, 2.0)),
                       layer(attention(16, 1, 32, 64, 0.16, (70, 1), (16, 30000.0), True), moe(16, 2, 128))], eps=1e-4)
# sizes that are multiples of nothing
G4 = config(101, 50, [layer(memory(5, 9, 13, 4.5), moe(7, 3, 9, 11)), layer(attention(3, 3, 22, 14, 0.22, (9, 4), (6, 777.0)), dense(45, 1.0)),
                      layer(memory(3, 10, 7, 12.0), moe(3, 2, 11)), layer(attention(2, 1, 10, 6, 0.3, (25, 0), (10, 60.0), True), moe(4, 1, 13, 21))],
            eps=1e-5)
CONFIGS = {"G1": G1, "G2": G2, "G3": G3, "G4": G4}
# no routed feed-forward: in bfloat16 no choice of experts can go the other way
DENSE = config(89, 64, [layer(memory(2, 16, 24, 7.0), dense(96, 1.1)), layer(attention(4, 1, 32, 48, 0.2, (24, 7), (32, 1000.0), True), dense(128, 2.0)),
                        layer(memory(4, 16, 32, 3.0)), layer(attention(6, 3, 16, 16, 0.25, (30, 17), (8, 40.0), True), dense(64, 0.7))])


def drawn(seed):
    """A configuration drawn from a seed: any order of layers, sizes that the tiled kernels take and sizes that they do not."""
    import random
    r = random.Random(seed)
    kv, vdim = r.choice([1, 2, 3]), r.choice([16, 24, 32, 48])

    def att(mix):
        g, dv = (kv, vdim) if mix else (r.choice([1, 2]), r.choice([8, 16, 20, 64]))
        dim = r.choice([16, 32, 48, 20, 64])
        mask = (r.choice([1, 13, 16, 40, 64]), r.choice([0, 1, 4, 16, 19, 50])) if r.random() < 0.8 else None
        rot = (r.choice([2, 8, dim]), r.choice([20.0, 1000.0, 1e6])) if r.random() < 0.8 else None
        return attention(g * r.choice([1, 2, 4]), g, dim, dv, r.uniform(0.5, 1.5) * dim ** -0.5, mask, rot, mix)

    def mem():
        return memory(r.choice([1, 2, 3, 6]), r.choice([8, 12, 32, 64, 96, 128, 10]), r.choice([8, 16, 24, 32, 64, 7]), r.uniform(1.0, 16.0))

    def mlp():
        kind = r.random()
        if kind < 0.2:
            return None
        if kind < 0.5:
            return dense(r.choice([48, 128, 256, 72]), r.uniform(0.3, 4.0))
        experts = r.choice([1, 4, 8, 12])
        return moe(experts, r.randint(1, experts), r.choice([16, 24, 64, 30]), r.choice([None, 32, 40, 128]))

    layers = [layer(att(r.random() < 0.7) if r.random() < 0.5 else mem(), mlp()) for _ in range(r.randint(2, 6))]
    return config(r.choice([61, 128, 200]), r.choice([64, 96, 128, 72]), layers, eps=r.choice([1e-6, 1e-5, 1e-4]))


def one_layer(mixer, width=48, vocab=61, mlp=None, eps=1e-6):
    return config(vocab, width, [layer(mixer, mlp)], eps=eps)


def lively_tensors(config, seed, dtype=torch.bfloat16, settled=False):
    """Weights at which every mechanism counts: matrices that keep activations of order one, forget gates spread over what
    keeps a state for a few tokens and for hundreds, sinks, shares of a mix and norm weights away from zero and one.
    `settled`: every token's embedding names its experts, layer by layer, on dimensions of their own that the routers read, so
    that rounding seldom changes a choice."""
    from fastmlx_b200 import registry
    cfg, model = registry.build_model(config)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for spec in model.weight_specs():
        t = torch.randn(spec.shape, generator=g, dtype=torch.float32)
        if spec.kind == "forget_bias":
            t = t * 1.5 + 2.5
        elif spec.kind == "share":
            t = torch.sigmoid(t) * 0.6 + 0.2
        elif spec.name.endswith(".sink"):
            t = t * 1.5
        elif spec.name.endswith(".router"):
            t = t * (0.1 if settled else 1.5) / shape_in(spec)
        elif spec.kind == "matrix":
            t = t / shape_in(spec)
        elif spec.kind == "embedding":
            t = t * 0.7
        elif spec.kind == "bias":
            t = t * 0.3
        elif spec.kind == "norm0":
            t = t * 0.2
        elif spec.kind == "norm":
            t = 1.0 + 0.2 * t
        out[spec.name] = t
    if settled:
        at, vocab = 0, config["vocab"]
        for i, spec in enumerate(config["layers"]):
            if not spec["mlp"] or spec["mlp"]["kind"] != "moe":
                continue
            E, top = spec["mlp"]["router"]["experts"], spec["mlp"]["router"]["top"]
            for e in range(E):
                out[f"l{i}.mlp.router"][e, at + e] = 3.0
            chosen = torch.zeros(vocab, E)
            chosen.scatter_(1, torch.rand(vocab, E, generator=g).argsort(1)[:, :top], 1.0)
            out["embed"][:, at:at + E] = (2 * chosen - 1) * (2.0 + 1.3 * torch.rand(vocab, E, generator=g))
            at += E
    return {n: t.to(dtype) for n, t in out.items()}


def shape_in(spec):
    return spec.shape[-1] ** 0.5


def make_model_dir(root, config, seed, tensors=None):
    """A folder with config.json and model.safetensors of lively weights (or of the tensors given)."""
    from fastmlx_b200.weights import safetensors_io as st
    d = os.path.join(str(root), f"gepadra_{config['vocab']}_{config['width']}_{len(config['layers'])}_{seed}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(config, f)
    st.write_file(os.path.join(d, "model.safetensors"), tensors if tensors is not None else lively_tensors(config, seed),
                  {"format": "pt"})
    return d
