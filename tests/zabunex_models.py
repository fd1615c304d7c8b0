"""Small Zabunex configurations and random weights for the tests, made here by the tensor naming rule itself (not from
the library's tensor lists), stored in bfloat16 as a model folder."""
import json
import os
import random

import torch


def attention(heads, kv_heads, dim, scale, bias_max, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "bias_max": bias_max}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m}


def left(heads, kv_heads, dim, vdim, conv, block, scale, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale}
    if block:
        m["mask"] = {"size": block}
    if rot:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
        if len(rot) > 2:
            m["rot"]["scaling"] = {"factor": rot[2]}
    return m


def right(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def parallel(a, b, left_scale, right_scale):
    return {"type": "parallel", "mixer": {"left": a, "right": b, "left_scale": left_scale, "right_scale": right_scale}}


def layer(mixer, ff=None):
    return {**mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Zabunex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# every size differs from every other: 3, 2 and 1 query heads per kv head, values wider and narrower than keys, blocks of 9, 33 and
# 130 positions over pages of 64, two, three and five taps, part of a head turned, all of it, nothing; groups shared by 2 and 3
# heads, norms in 1, 3 and 4 parts; a bias that reaches 20, 90 and 300 positions; layers without a feed-forward
MIXED = config(64, 97, [
    layer(parallel(left(6, 2, 16, 12, 3, 33, 0.3, (8, 100.0, 2.0)), right(4, 8, 10, 2, 4, 4), 0.7, 1.3), 72),
    layer(attention(4, 2, 20, 0.25, 90, (0.4, 25)), 104),
    layer(attention(3, 1, 24, 0.2, 20)),
    layer(parallel(left(2, 2, 14, 22, 2, 9, 0.35), right(6, 6, 24, 2, 5, 3), 1.1, 0.6)),
    layer(parallel(left(4, 1, 12, 16, 4, 130, 0.3, (12, 1000.0, 4.0)), right(3, 20, 36, 1, 2, 1), 0.5, 0.9), 88),
    layer(attention(5, 5, 8, 0.5, 300, (0.2, 64)), 56),
])
# a width that no tensor-core product takes, sizes that are no multiples of 4 or 8, one head, one tap on either side (no state of a
# convolution), blocks of one page and of 70, no block mask at all, an odd number of columns in every product
ODD = config(44, 61, [
    layer(attention(1, 1, 10, 0.3, 40, (0.5, 7)), 36),
    layer(parallel(left(3, 3, 9, 7, 1, 64, 0.3), right(3, 7, 13, 3, 3, 7), 1.0, 1.0), 50),
    layer(parallel(left(4, 2, 6, 11, 5, 70, 0.4, (4, 37.0, 3.0)), right(5, 9, 6, 1, 1, 5), 0.3, 1.7)),
    layer(attention(4, 2, 7, 0.35, 150), 42),
    layer(parallel(left(2, 1, 11, 5, 2, None, 0.3, (2, 500.0)), right(1, 34, 65, 1, 7, 2), 0.8, 0.4), 38),
], eps=1e-6)
# sizes of the tensor-core kernels: heads of 64 and 128 channels (equal and unlike values), blocks of 130 and 200 positions, states of
# 64 and 128 channels
WIDE = config(128, 83, [
    layer(parallel(left(6, 2, 64, 128, 4, 130, 0.13, (32, 10000.0, 2.0)), right(4, 32, 64, 2, 4, 2), 0.9, 0.8), 256),
    layer(attention(6, 3, 64, 0.12, 128, (0.3, 100)), 192),
    layer(attention(2, 2, 128, 0.1, 250, (0.1, 64)), 136),
    layer(parallel(left(3, 1, 128, 64, 3, 200, 0.09, (128, 500000.0, 8.0)), right(2, 64, 128, 1, 4, 1), 1.2, 0.5), 320),
])
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}


def bias_rows(L) -> int:
    """Rows of an attention layer's bias table (only the tensor's shape gives them): even numbers from 4 to 32."""
    return 4 + 2 * (int(L["mixer"]["bias_max"]) // 10 % 15)


def tensor_shapes(cfg):
    """name -> (shape, kind of values) by the naming rule."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": ((V, W), "embed"), "final.norm": ((W,), "norm"), "head": ((V, W), "head")}

    def heads(p, m, conv):
        q, k, v, o = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]
        for name, n in (("q", q), ("k", k), ("v", v)):
            if name == "v" and not conv:
                continue
            out[p + name] = ((n, W), "linear")
            if conv:
                out[p + name + ".conv"] = ((n, conv), "conv")
        out[p + "q.norm"], out[p + "k.norm"], out[p + "o"] = ((q,), "norm"), ((k,), "norm"), ((W, o), "linear")

    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", L["mixer"], L.get("mlp")
        out[p + "norm1"] = ((W,), "norm")
        if L["type"] == "attention":
            heads(p + "mix.", m, None)
            out[p + "mix.rel"] = ((bias_rows(L), m["heads"]), "rel")
        else:
            heads(p + "mix.left.", m["left"], m["left"]["conv"])
            r, q = m["right"], p + "mix.right."
            inner, channels = r["heads"] * r["vdim"], r["heads"] * r["vdim"] + 2 * r["groups"] * r["state"]
            out[q + "in"] = ((inner + channels + r["heads"], W), "linear")
            out[q + "conv"], out[q + "conv.b"] = ((channels, r["conv"]), "conv"), ((channels,), "bias")
            out[q + "dt_bias"], out[q + "A_log"], out[q + "D"] = ((r["heads"],), "step"), ((r["heads"],), "rate"), ((r["heads"],), "norm")
            out[q + "norm"], out[q + "o"] = ((inner,), "norm"), ((W, inner), "linear")
        if f:
            out[p + "norm2"] = ((W,), "norm")
            out[p + "mlp.up"], out[p + "mlp.down"] = ((f["ff"], W), "linear"), ((W, f["ff"]), "linear")
    return out


def random_weights(cfg, seed):
    """name -> bfloat16 tensor, of the order a trained model has, so that every mechanism moves the logits: bias tables of
    the size of the scores, decays that keep a state for tens of tokens, taps of either sign, norm weights away from one."""
    gen = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=gen)
        t = {"linear": lambda: r * (1.0 / shape[-1] ** 0.5), "embed": lambda: r * 0.8, "head": lambda: r * (2.0 / W ** 0.5),
             "norm": lambda: 1.0 + 0.3 * r, "bias": lambda: 0.4 * r, "rel": lambda: 1.2 * r, "conv": lambda: r * (1.0 / shape[-1] ** 0.5),
             "step": lambda: -1.0 + 0.5 * r, "rate": lambda: -2.0 + 0.8 * r}[kind]()
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(folder, cfg, seed, weights=None):
    from camelid_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    weights = weights if weights is not None else random_weights(cfg, seed)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), weights)
    return weights


def as_float64(weights):
    return {k: v.to(torch.float64).numpy() for k, v in weights.items()}


def random_config(seed, tensor_cores=False):
    """A configuration drawn from a seed: sizes, head counts, order and number of layers, blocks, taps, turned channels, groups, bias
    reach, temperatures and scales all vary; small enough for the plain implementation. ``tensor_cores``: heads and states
    that the bfloat16 tensor-core kernels take."""
    rng = random.Random(seed if not tensor_cores else 1000 + seed)

    def heads():
        g = rng.randint(1, 3)
        return g * rng.randint(1, 3), g

    layers = []
    for i in range(rng.randint(3, 5)):
        ff = rng.choice([None, 24, 52, 88, 120])
        h, g = heads()
        scale = rng.uniform(0.08, 0.15) if tensor_cores else rng.uniform(0.15, 0.4)
        if rng.random() < 0.5:
            dim = rng.choice([64, 128]) if tensor_cores else rng.randint(3, 24)
            layers.append(layer(attention(h, g, dim, scale, rng.choice([17, 33, 64, 100, 200.5]),
                                          rng.choice([None, (0.3, 16), (0.1, 50), (0.5, 3)])), ff))
            continue
        dim, vdim = (rng.choice([64, 128]), rng.choice([64, 128])) if tensor_cores else (rng.randint(3, 24), rng.randint(3, 24))
        rot = rng.choice([None, (2 * rng.randint(1, dim // 2), rng.choice([37.0, 10000.0])),
                          (2 * rng.randint(1, dim // 2), 500000.0, rng.uniform(1.5, 8.0))])
        a = left(h, g, dim, vdim, rng.randint(1, 5), rng.choice([None, 1, 5, 63, 64, 65, 100]), scale, rot)
        groups = rng.randint(1, 3)
        ssm = groups * rng.randint(1, 3)
        P = rng.choice([16, 32, 64]) if tensor_cores else rng.randint(2, 24)
        parts = [n for n in range(1, 7) if ssm * P % n == 0]
        b = right(ssm, P, rng.choice([16, 64, 128]) if tensor_cores else rng.randint(2, 70), groups, rng.randint(1, 6), rng.choice(parts))
        layers.append(layer(parallel(a, b, rng.uniform(0.3, 1.5), rng.uniform(0.3, 1.5)), ff))
    return config(rng.choice([64, 128]) if tensor_cores else rng.choice([40, 48, 70, 96]), rng.randint(50, 120), layers,
                  eps=rng.choice([1e-5, 1e-6]))
