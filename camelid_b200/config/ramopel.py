"""The Ramopel decoder's config.json as a typed configuration, and its plan.

Both sublayers of a layer read the same stream, x += mixer(norm1(x)) + ff(norm2(x)), with RMS norms whose weights are
stored around zero (x / rms(x) * (1 + w)). The layers take one of two mixers in the order ``layers`` gives:

* ``latent_attention``: queries made from a normed latent of ``q_rank`` channels; all heads' keys and values are maps of
  one normed latent row of ``kv_rank`` channels per position plus one turned key part of ``rot_dim`` channels shared by
  the heads (pairs of neighbouring channels); a window of ``mask.size`` keys; an ordinary softmax. A layer with
  ``kv_from`` j reads the latent rows layer j's cache holds, with maps, queries and a window of its own;
* ``general_delta``: the delta rule with a decay and a removal rate per key channel on a float32 state per sequence.

A layer's feed-forward is dense (the activation is a weighted sum of a row's normed powers), a mixture of gated experts
(softmax over the chosen logits; a shared expert with an output gate of one number per token), or absent. Rows start as
embed[token] * ``embedding.scale``; the logits are head(final norm(x)).

Keys read (all sizes and constants come from here): ``architecture``, ``vocab``, ``width``, ``norm.eps``,
``embedding.scale``, ``layers[i].type``; of ``layers[i].mixer``: latent_attention ``{heads, dim, rot_dim, vdim, kv_rank,
q_rank, scale, mask.size, rot.{base, dims}, kv_from}``, general_delta ``{heads, dim}``; ``layers[i].mlp`` null,
``{kind: "dense", ff}`` or ``{kind: "moe", router.{experts, top}, expert.{ff, limit}, shared.{ff, limit}}``. Missing: ``mask``
(all earlier keys), ``kv_from`` (rows of its own), ``vdim`` (``dim``), ``shared`` (none), ``embedding.scale`` (1). The width
of the decays' narrow input (``w1``, ``w2``) is the stored tensors' own; ``mixer.rank`` is this library's own optional key
for models with random weights.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from ..errors import ConfigError
from .fomatar import NO_POSITION_LIMIT, _get, _positive
from .plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

MIXERS = ("latent_attention", "general_delta")
GATE_SLOPE, UP_SHIFT = 1.702, 1.0           # the experts' activation: min(g, limit) sigmoid(1.702 g) (clamp(u) + 1)


def _latent(m: dict, w: str) -> dict:
    out = {"heads": _positive(m, "heads", w), "dim": _positive(m, "dim", w)}
    out["vdim"] = _positive(m, "vdim", w, out["dim"])
    for k in ("rot_dim", "kv_rank", "q_rank"):
        out[k] = _positive(m, k, w)
    out["scale"] = _get(m, "scale", w, float)
    mask = _get(m, "mask", w, None, None)
    out["window"] = _positive(mask, "size", w + ".mask") if mask is not None else None
    rot = _get(m, "rot", w)
    out["base"], dims = _get(rot, "base", w + ".rot", float), _get(rot, "dims", w + ".rot", int)
    if dims != out["rot_dim"] or dims % 2:
        raise ConfigError(w + ".rot.dims", f"must be even and equal rot_dim ({out['rot_dim']}), got {dims}")
    if out["base"] <= 0:
        raise ConfigError(w + ".rot.base", f"must be greater than zero, got {out['base']}")
    out["kv_from"] = _get(m, "kv_from", w, int, None)
    return out


def _expert(d: dict, w: str) -> dict:
    limit = _get(d, "limit", w, float)
    if limit <= 0:
        raise ConfigError(w + ".limit", f"must be greater than zero, got {limit}")
    return {"ff": _positive(d, "ff", w), "limit": limit}


def _feed_forward(mlp, w: str):
    if mlp is None:
        return None
    kind = _get(mlp, "kind", w)
    if kind == "dense":
        return {"kind": kind, "ff": _positive(mlp, "ff", w)}
    if kind != "moe":
        raise ConfigError(w + ".kind", f"unknown feed-forward {kind!r}; known: dense, moe")
    router = _get(mlp, "router", w)
    out = {"kind": kind, "experts": _positive(router, "experts", w + ".router"), "top": _positive(router, "top", w + ".router"),
           "expert": _expert(_get(mlp, "expert", w), w + ".expert"), "shared": None}
    if out["top"] > out["experts"]:
        raise ConfigError(w + ".router.top", f"each token picks 1..{out['experts']} experts, got {out['top']}")
    shared = _get(mlp, "shared", w, None, None)
    if shared is not None:
        out["shared"] = _expert(shared, w + ".shared")
    return out


def _check_borrowed(layers: list) -> None:
    for i, L in enumerate(layers):
        j = L["mixer"].get("kv_from")
        if j is None:
            continue
        w = f"layers[{i}].mixer.kv_from"
        if not 0 <= j < i or layers[j]["type"] != "latent_attention":
            raise ConfigError(w, f"must name an earlier latent_attention layer, got {j}")
        src = layers[j]["mixer"]
        if src["kv_from"] is not None:
            raise ConfigError(w, f"layer {j} has no latent rows of its own")
        for k in ("kv_rank", "rot_dim", "base"):
            if src[k] != L["mixer"][k]:
                raise ConfigError(w, f"layer {j} has another {k} ({src[k]}) than this layer ({L['mixer'][k]})")


@dataclass(frozen=True)
class RamopelConfig:
    raw: dict
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple                   # dicts: type, mixer (validated), mlp

    @classmethod
    def from_dict(cls, d: dict) -> "RamopelConfig":
        vocab, width = _positive(d, "vocab", ""), _positive(d, "width", "")
        eps = _get(_get(d, "norm", ""), "eps", "norm", float)
        emb_scale = _get(_get(d, "embedding", "", None, None) or {}, "scale", "embedding", float, 1.0)
        raw_layers = _get(d, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers", "must be a list with at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            w = f"layers[{i}]"
            kind = _get(L, "type", w)
            if kind not in MIXERS:
                raise ConfigError(w + ".type", f"unknown layer type {kind!r}; known: {', '.join(MIXERS)}")
            m, wm = _get(L, "mixer", w), w + ".mixer"
            if kind == "latent_attention":
                mixer = _latent(m, wm)
            else:
                mixer = {"heads": _positive(m, "heads", wm), "dim": _positive(m, "dim", wm), "rank": _positive(m, "rank", wm, None)}
            layers.append({"type": kind, "mixer": mixer, "mlp": _feed_forward(L.get("mlp"), w + ".mlp")})
        _check_borrowed(layers)
        return cls(copy.deepcopy(d), vocab, width, eps, emb_scale, tuple(layers))

    def to_dict(self) -> dict:
        return copy.deepcopy(self.raw)

    @property
    def stop_token_ids(self) -> tuple:
        return ()


def _cache_window(layers, i: int):
    """How far back the latent rows of layer i must reach: the widest view of the layer itself and of those that read
    its rows (0: all positions)."""
    views = [layers[i]["mixer"]["window"]] + [L["mixer"]["window"] for L in layers if L["mixer"].get("kv_from") == i]
    return 0 if None in views else max(views)


def ramopel_plan(cfg: RamopelConfig) -> ModelPlan:
    """Parts per layer (tensor names ``l<i>.…``); every layer runs once, in order; a layer with borrowed latent rows names
    its source in the schedule."""
    norm = {"hidden_size": cfg.width, "eps": cfg.eps, "offset": 1.0}
    layers, schedule = [], []
    for i, L in enumerate(cfg.layers):
        p, m, f = f"l{i}.", L["mixer"], L["mlp"]
        common = {"hidden_size": cfg.width, "eps": cfg.eps, "num_heads": m["heads"]}
        if L["type"] == "latent_attention":
            borrowed = m["kv_from"] is not None
            mixer = PartSpec("latent_attention", {
                **common, "head_dim": m["dim"], "rot_dim": m["rot_dim"], "value_dim": m["vdim"], "rank": m["kv_rank"],
                "q_rank": m["q_rank"], "scale": m["scale"], "window": m["window"], "borrow_rows": borrowed,
                "cache_window": m["window"] if borrowed else _cache_window(cfg.layers, i),
                "position": PartSpec("rope", {"rotary_dim": m["rot_dim"], "theta": m["base"], "scaling": None,
                                              "pairing": "interleaved"})}, p + "mix.")
        else:
            mixer = PartSpec("general_delta", {**common, "key_dim": m["dim"], "value_dim": m["dim"], "rank": m["rank"]}, p + "mix.")
        ffn = None
        if f is not None and f["kind"] == "dense":
            ffn = PartSpec("dense", {"hidden_size": cfg.width, "intermediate_size": f["ff"], "activation": "poly_norm",
                                     "eps": cfg.eps}, p + "mlp.")
        elif f is not None:
            sh = f["shared"]
            ffn = PartSpec("routed_experts", {
                "hidden_size": cfg.width, "experts": f["experts"], "top": f["top"], "expert_size": f["expert"]["ff"],
                "scoring": "softmax", "renormalize": True, "router_bias": True,
                "gate_act": (GATE_SLOPE, f["expert"]["limit"], UP_SHIFT),
                "shared_size": sh["ff"] if sh else None, "shared_output_gate": sh is not None,
                "shared_gate_act": (GATE_SLOPE, sh["limit"], UP_SHIFT) if sh else None}, p + "mlp.")
        layers.append(LayerSpec(
            arrangement="parallel",
            norm1=PartSpec("rmsnorm", {**norm, "tensor": p + "norm1"}),
            mixer=mixer,
            norm2=PartSpec("rmsnorm", {**norm, "tensor": p + "norm2"}) if ffn is not None else None,
            ffn=ffn,
        ))
        schedule.append(ScheduleEntry(i, cache_source=m.get("kv_from")))
    return ModelPlan(
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tensor": "embed",
                                         "scale": cfg.embedding_scale}),
        layers=tuple(layers),
        schedule=tuple(schedule),
        final_norm=PartSpec("rmsnorm", {**norm, "tensor": "final.norm"}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": None, "tensor": "head"}),
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_position=NO_POSITION_LIMIT,
        stop_token_ids=(),
    )
