"""Small Ramopel configurations and random weights for the tests, made here by the tensor naming rule itself (not from
the library's tensor lists), stored in bfloat16 as a model folder."""
import json
import os
import random

import torch


def latent(heads, dim, rot_dim, vdim, rank, q_rank, window, base, scale, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m}


def delta(heads, dim):
    return {"type": "general_delta", "mixer": {"heads": heads, "dim": dim}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, shared=None):
    m = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    return m


def layer(mixer, mlp=None):
    return {**mixer, "mlp": mlp}


def config(width, vocab, layers, emb=1.0, eps=1e-5):
    return {"architecture": "Ramopel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "layers": layers}


# every size differs from every other; a borrower that sees further back than its source, another that sees less, a
# mixer of either kind before either kind of feed-forward and before none
MIXED = config(64, 97, [
    layer(latent(3, 16, 8, 12, 40, 24, 9, 100.0, 0.25), dense(72)),
    layer(delta(2, 24), moe(7, 2, 24, 0.8, (56, 0.6))),
    layer(latent(5, 12, 8, 20, 40, 32, 33, 100.0, 0.3, kv_from=0), moe(5, 3, 32, 1.5)),
    layer(delta(3, 16)),
    layer(latent(2, 20, 8, 28, 40, 48, 5, 100.0, 0.2, kv_from=0)),
    layer(delta(4, 8), dense(104)),
], emb=3.0)
# a width that no tensor-core product takes, sizes that are no multiples of 8, one head, one choice, a latent layer that
# sees everything and lends its rows to one with a window longer than a page, a narrow input of 6 channels
ODD = config(44, 61, [
    layer(delta(3, 10), dense(36)),
    layer(latent(1, 10, 6, 7, 18, 14, None, 500.0, 0.3), moe(6, 1, 10, 2.0, (20, 1.0))),
    layer(latent(4, 9, 6, 11, 18, 22, 70, 500.0, 0.35, kv_from=1), dense(50)),
    layer(delta(1, 34), moe(3, 3, 14, 0.7)),
    layer(latent(2, 6, 4, 5, 13, 9, 64, 37.0, 0.4)),
], emb=1.0, eps=1e-6)
# sizes of the tensor-core kernels: latents of 96 and 32 channels, windows of 130 and 64 over pages of 64, state heads of
# 64 and 128 channels, every routed layer's rows use all of its experts (no choice that rounding could turn)
WIDE = config(128, 83, [
    layer(latent(4, 32, 16, 48, 96, 64, 130, 10000.0, 0.14), dense(256)),
    layer(delta(2, 64), moe(4, 4, 64, 1.2, (128, 0.9))),
    layer(latent(6, 24, 16, 32, 96, 40, 200, 10000.0, 0.16, kv_from=0), dense(192)),
    layer(delta(1, 128), moe(3, 3, 48, 2.0, (80, 1.5))),
    layer(latent(3, 16, 32, 24, 32, 56, 64, 1000.0, 0.15), dense(136)),
], emb=2.0)
CONFIGS = {"mixed": MIXED, "odd": ODD, "wide": WIDE}


def narrow_size(L) -> int:
    """Width of the decays' narrow input of a delta layer (only the tensors' shapes give it)."""
    return 4 + L["mixer"]["dim"] % 7 * 2


def tensor_shapes(cfg):
    """name -> (shape, kind of values) by the naming rule."""
    W, V = cfg["width"], cfg["vocab"]
    out = {"embed": ((V, W), "embed"), "final.norm": ((W,), "norm0"), "head": ((V, W), "head")}
    for i, L in enumerate(cfg["layers"]):
        p, q, m, f = f"l{i}.", f"l{i}.mix.", L["mixer"], L.get("mlp")
        H, D = m["heads"], m["dim"]
        out[p + "norm1"] = ((W,), "norm0")
        if L["type"] == "latent_attention":
            R, C, Q, Dv = m["rot_dim"], m["kv_rank"], m["q_rank"], m["vdim"]
            out[q + "dq"], out[q + "dq.norm"], out[q + "uq"] = ((Q, W), "linear"), ((Q,), "norm"), ((H * (D + R), Q), "linear")
            if m.get("kv_from") is None:
                out[q + "dkv"], out[q + "dkv.norm"] = ((C + R, W), "linear"), ((C,), "norm")
            out[q + "uk"], out[q + "uv"], out[q + "o"] = ((H * D, C), "linear"), ((H * Dv, C), "linear"), ((W, H * Dv), "linear")
        else:
            n = narrow_size(L)
            for name in "rkvag":
                out[q + name] = ((H * D, W), "gate" if name in "ag" else "linear")
            out[q + "a.b"], out[q + "w0"] = ((H * D,), "bias"), ((H * D,), "bias")
            out[q + "w1"], out[q + "w2"] = ((n, W), "linear"), ((H * D, n), "gate")
            out[q + "norm"], out[q + "o"] = ((H * D,), "norm"), ((W, H * D), "linear")
        if not f:
            continue
        out[p + "norm2"] = ((W,), "norm0")
        g = p + "mlp."
        if f["kind"] == "dense":
            out[g + "up"], out[g + "down"], out[g + "act"] = ((f["ff"], W), "linear"), ((W, f["ff"]), "linear"), ((4,), "poly")
            continue
        E = f["router"]["experts"]
        out[g + "router"], out[g + "router.b"] = ((E, W), "gate"), ((E,), "bias")
        sizes = [(f"e{e}.", f["expert"]["ff"]) for e in range(E)]
        if f.get("shared"):
            sizes.append(("shared.", f["shared"]["ff"]))
            out[g + "shared.sg"] = ((1, W), "gate")
        for name, ff in sizes:
            out[g + name + "gate"], out[g + name + "up"], out[g + name + "down"] = ((ff, W), "linear"), ((ff, W), "linear"), ((W, ff), "linear")
    return out


def random_weights(cfg, seed):
    """name -> bfloat16 tensor, of the order a trained model has, so that every mechanism moves the logits: norm weights
    around zero and around one, gates away from one half, biases, all four numbers of the activation."""
    gen = torch.Generator().manual_seed(seed)
    W = cfg["width"]
    out = {}
    for name, (shape, kind) in tensor_shapes(cfg).items():
        r = torch.randn(shape, generator=gen)
        t = {"linear": lambda: r * (1.0 / shape[-1] ** 0.5), "gate": lambda: r * (2.0 / shape[-1] ** 0.5),
             "embed": lambda: r * 0.8, "head": lambda: r * (4.0 / W ** 0.5), "norm": lambda: 1.0 + 0.3 * r,
             "norm0": lambda: 0.3 * r, "bias": lambda: 0.5 * r,
             "poly": lambda: torch.tensor([0.6, -0.35, 0.25, 0.1]) + 0.1 * r}[kind]()
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
    """A configuration drawn from a seed: sizes, head counts, order and number of layers, windows, borrowed rows,
    feed-forwards, limits and constants all vary; small enough for the plain implementation. ``tensor_cores``: widths and
    latents that the bfloat16 tensor-core kernels take, and no choice of experts that rounding could turn."""
    rng = random.Random(seed if not tensor_cores else 1000 + seed)
    even = lambda lo, hi: 2 * rng.randint(lo // 2, hi // 2)      # noqa: E731

    def mlp():
        kind = rng.choice([None, "dense", "dense", "moe", "moe"])
        if kind is None:
            return None
        if kind == "dense":
            return dense(rng.choice([24, 52, 88, 120]))
        experts = rng.randint(2, 9)
        ff = rng.choice([16, 48] if tensor_cores else [10, 16, 33, 48])
        shared = (rng.choice([24, 64, 40]), rng.uniform(0.5, 2.0)) if rng.random() < 0.7 else None
        return moe(experts, experts if tensor_cores else rng.randint(1, experts), ff, rng.uniform(0.5, 2.0), shared)

    layers, sources = [], []
    for i in range(rng.randint(3, 6)):
        if i == 0 or rng.random() < 0.5:
            heads, dim, vdim = rng.randint(1, 6), rng.randint(3, 24), rng.randint(3, 24)
            window, q_rank = rng.choice([None, 1, 3, 17, 64, 65, 100]), rng.choice([8, 15, 24, 40])
            scale = rng.uniform(0.1, 0.4)
            if sources and rng.random() < 0.6:
                j, rd, rank, base = rng.choice(sources)
                layers.append(layer(latent(heads, dim, rd, vdim, rank, q_rank, window, base, scale, kv_from=j), mlp()))
                continue
            rd, rank = (rng.choice([16, 32]), rng.choice([32, 64, 96, 128])) if tensor_cores else (even(2, 16), rng.choice([8, 20, 32, 63]))
            base = rng.choice([37.0, 1000.0, 250000.0])
            sources.append((i, rd, rank, base))
            layers.append(layer(latent(heads, dim, rd, vdim, rank, q_rank, window, base, scale), mlp()))
        else:
            layers.append(layer(delta(rng.randint(1, 4), rng.choice([16, 32, 64]) if tensor_cores else rng.randint(3, 40)), mlp()))
    return config(rng.choice([64, 128]) if tensor_cores else rng.choice([40, 48, 70, 96]), rng.randint(50, 120), layers,
                  emb=rng.choice([1.0, 0.5, 12.0]), eps=rng.choice([1e-5, 1e-6]))
