"""Small Bonerax configurations for the tests: they differ from one another in every size and option, and use values that a
usual model makes equal or 1 (one head, as many kv heads as heads or fewer, values narrower, wider or as wide as keys, one
convolution tap or many, a tau of 1, a scale of zero or below, a rotation over the whole head, over a part or none, YaRN
or plain frequencies, no window or one of a single token, one chosen expert or all, no feed-forward, layers that use another
one's weights, no cap on the logits), and weights of a size at which every mechanism matters."""
import json
import os

import torch


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def attention(heads, kv_heads, dim, vdim, scale, window=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if rot is not None:
        m["rot"] = rot
    return m


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def gla(heads, dim, vdim, tau):
    return {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def pair(left, right, left_scale, right_scale):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(kind, mixer, mlp=None, weights_of=None):
    d = {"type": kind, "mixer": mixer, "mlp": mlp}
    if weights_of is not None:
        d["weights_of"] = weights_of
    return d


def again(layers, j):
    return dict(layers[j], weights_of=j)


def config(vocab, width, layers, eps=1e-6, scale=None, cap=None):
    c = {"architecture": "Bonerax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if scale is not None:
        c["logit_scale"] = scale
    if cap is not None:
        c["logit_softcap"] = cap
    return c


_p1 = layer("parallel", pair(attention(4, 2, 16, 32, 0.3, window=19, rot=rot(8, 500.0, (4.0, 96, 8.0, 1.5))),
                             delta(4, 2, 12, 20, 3), 1.25, -0.6), moe(6, 2, 24))
_d1 = layer("channel_delta", delta(6, 2, 24, 16, 4), dense(96))
B1 = config(211, 96, [_p1, layer("gla", gla(3, 20, 12, 5.0), moe(5, 5, 16)), _d1, again([_p1, None, _d1], 0), again([None, None, _d1], 2),
                      layer("gla", gla(2, 8, 40, 1.0))], scale=0.7, cap=11.0)
B2 = config(97, 64, [layer("channel_delta", delta(1, 1, 64, 8, 1)),
                     layer("parallel", pair(attention(2, 2, 32, 32, 0.2, window=1), delta(2, 2, 8, 32, 2), 0.5, 1.5), dense(128)),
                     layer("parallel", pair(attention(3, 1, 16, 16, 0.25, rot=rot(16, 50.0)), delta(3, 1, 16, 24, 5), 0.0, 1.0), moe(3, 1, 32))],
            eps=1e-5)
# sizes that the tiled kernels and the blocked products take: heads in steps of 16, feed-forwards in blocks of 128
_p3 = layer("parallel", pair(attention(8, 2, 64, 32, 0.125, window=33, rot=rot(64, 250000.0, (3.0, 128, 16.0, 1.0))),
                             delta(4, 4, 64, 64, 4), 0.9, 0.4), dense(256))
B3 = config(130, 128, [layer("gla", gla(4, 64, 64, 16.0), moe(8, 3, 64)), _p3,
                       layer("channel_delta", delta(2, 2, 128, 128, 4), moe(4, 2, 128)), again([None, _p3], 1),
                       layer("parallel", pair(attention(16, 1, 32, 64, 0.11, window=70, rot=rot(16, 30000.0)), delta(2, 1, 96, 48, 6), 1.0, 1.0))],
            eps=1e-4, scale=3.0, cap=25.0)
# sizes that are multiples of nothing
B4 = config(101, 50, [layer("parallel", pair(attention(3, 3, 22, 14, 0.22, window=9, rot=rot(6, 777.0, (2.0, 40, 6.0, 1.0))),
                                             delta(3, 3, 7, 5, 4), 0.3, 2.0), moe(7, 3, 9)),
                      layer("gla", gla(5, 9, 13, 3.5), dense(45)), layer("channel_delta", delta(3, 1, 10, 18, 3), moe(3, 2, 11))],
            eps=1e-5, cap=6.0)
CONFIGS = {"B1": B1, "B2": B2, "B3": B3, "B4": B4}


def one_layer(kind, mixer, width=48, vocab=61, mlp=None, eps=1e-6):
    return config(vocab, width, [layer(kind, mixer, mlp)], eps=eps)


def ranks(name, width):
    """The ranks that the tests' weights give the low-rank projections: odd ones too, and not the parts' own default."""
    return {"a1": 5, "g1": 12}[name] if width % 16 else {"a1": 8, "g1": 24}[name]


def lively_tensors(config, seed, dtype=torch.bfloat16, settled=False):
    """Weights at which every mechanism counts: matrices that keep activations of order one, decays spread over (0, 1), norm
    weights and biases away from one and zero.  `settled`: routers whose biases decide more and whose inputs decide less,
    so that rounding seldom changes a choice."""
    from fastmlx_b200 import registry
    from fastmlx_b200.parts import FreeDim
    cfg, model = registry.build_model(config)
    g = torch.Generator().manual_seed(seed)
    out = {}
    for spec in model.weight_specs():
        shape = tuple(ranks(s.key.rsplit(".", 1)[1], cfg.width) if isinstance(s, FreeDim) else s for s in spec.shape)
        t = torch.randn(shape, generator=g, dtype=torch.float32)
        if spec.kind == "conv":
            t = t * 0.5
        elif spec.kind == "log_rate":
            t = torch.log(torch.sigmoid(t) * 0.98 + 0.02)
        elif spec.kind == "rate_bias":
            t = t * 0.8 - 1.0
        elif spec.name.endswith(".a2.b"):
            t = t * 1.5 + 2.0
        elif spec.name.endswith(".router.b"):
            t = t * (2.0 if settled else 0.5)
        elif spec.name.endswith(".router"):
            t = t * (0.2 if settled else 1.5) / shape[-1] ** 0.5
        elif spec.kind == "matrix":
            t = t / shape[-1] ** 0.5
        elif spec.kind == "embedding":
            t = t * 0.7
        elif spec.kind == "bias":
            t = t * 0.3
        elif spec.kind == "norm":
            t = 1.0 + 0.2 * t
        out[spec.name] = t.to(dtype)
    return out


def make_model_dir(root, config, seed, tensors=None):
    """A folder with config.json and model.safetensors of lively weights (or of the tensors given)."""
    from fastmlx_b200.weights import safetensors_io as st
    d = os.path.join(str(root), f"bonerax_{config['vocab']}_{config['width']}_{len(config['layers'])}_{seed}")
    os.makedirs(d, exist_ok=True)
    with open(os.path.join(d, "config.json"), "w") as f:
        json.dump(config, f)
    st.write_file(os.path.join(d, "model.safetensors"), tensors if tensors is not None else lively_tensors(config, seed),
                  {"format": "pt"})
    return d
# no routed feed-forward: in bfloat16 no choice of experts can go the other way
DENSE = config(89, 64, [layer("gla", gla(2, 16, 24, 4.0), dense(96)),
                        layer("parallel", pair(attention(4, 1, 32, 48, 0.2, window=24, rot=rot(32, 1000.0, (2.0, 64, 8.0, 1.0))),
                                               delta(2, 2, 32, 16, 4), 0.7, 1.1), dense(128)),
                        layer("channel_delta", delta(4, 2, 16, 32, 3), dense(64))], scale=1.5, cap=20.0)
