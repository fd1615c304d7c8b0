"""The Zabunex decoder's config.json as a typed configuration, and its plan.

The sublayers of a layer read the stream itself and only their outputs are normed, x += norm1(mixer(x)) and
x += norm2(ff(x)) with RMS norms. The layers take one of two mixers in the order ``layers`` gives:

* ``attention``: grouped queries whose values are the keys' projection before its norm; RMS norms of q and of k over their
  whole projections; q times 1 + coef ln(floor((position + 1) / every) + 1); a learned bias per head on bucketed distances
  added to the scaled score; every earlier key is seen; the softmax denominator holds one more term exp(0);
* ``parallel``: two mixers side by side, ``left_scale`` * left + ``right_scale`` * right. Left: attention over blocks of
  ``mask.size`` positions with short convolutions on q, k and v, norms over the whole projections and a rotation of the first
  ``rot.dims`` channels of every head (pairs of halves; frequencies divided by ``rot.scaling.factor``). Right: a state-space
  recurrence with one decay per head and token, its inputs through a short convolution with bias and SiLU, its read-out times
  silu(z) and normed in ``norm_groups`` parts.

The feed-forward is dense with the square of ReLU, or absent. Rows start as embed[token]; the logits are head(final norm(x)).

Keys read (all sizes and constants come from here): ``architecture``, ``vocab``, ``width``, ``norm.eps``, ``layers[i].type``,
``layers[i].mlp`` null or ``{kind: "dense", ff}``, and of ``layers[i].mixer``: attention ``{dim, vdim, heads, kv_heads, scale,
bias_max, q_temp.{coef, every}}``; parallel ``left.{dim, vdim, heads, kv_heads, conv, scale, mask.size, rot.{dims, base,
scaling.factor}}``, ``right.{heads, vdim, state, groups, conv, norm_groups}``, ``left_scale``, ``right_scale``. Missing: ``vdim``
(``dim``; the right side's is required), ``kv_heads`` (``heads``), ``q_temp`` (none), ``mask`` (all earlier keys), ``rot`` (no
rotation), ``rot.scaling`` (1), ``groups`` and ``norm_groups`` (1), the two scales (1). The rows of a bias table are the stored
tensor's own; ``mixer.bias_rows`` is this library's own optional key for models with random weights.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from ..errors import ConfigError
from .fomatar import NO_POSITION_LIMIT, _get, _positive
from .plan import LayerSpec, ModelPlan, PartSpec, ScheduleEntry

MIXERS = ("attention", "parallel")


def _heads(m: dict, w: str) -> dict:
    out = {"heads": _positive(m, "heads", w), "dim": _positive(m, "dim", w)}
    out["vdim"] = _positive(m, "vdim", w, out["dim"])
    out["kv_heads"] = _positive(m, "kv_heads", w, out["heads"])
    if out["heads"] % out["kv_heads"]:
        raise ConfigError(w + ".kv_heads", f"{out['kv_heads']} does not divide {out['heads']} heads")
    out["scale"] = _get(m, "scale", w, float)
    return out


def _rot(m: dict, w: str, dim: int):
    """The ``rot`` entry of a mixer as the parameters of a rotary position part (None: no rotation)."""
    rot = _get(m, "rot", w, None, None)
    if rot is None:
        return None
    w += ".rot"
    dims, base = _get(rot, "dims", w, int), _get(rot, "base", w, float)
    if dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(w + ".dims", f"must be even and at most {dim}, got {dims}")
    if base <= 0:
        raise ConfigError(w + ".base", f"must be greater than zero, got {base}")
    scaling = _get(rot, "scaling", w, None, None)
    factor = _get(scaling, "factor", w + ".scaling", float) if scaling is not None else 1.0
    if factor <= 0:
        raise ConfigError(w + ".scaling.factor", f"must be greater than zero, got {factor}")
    if dims == 0:
        return None
    return {"rotary_dim": dims, "theta": base, "scaling": {"rope_type": "linear", "factor": factor}, "pairing": "split"}


def _attention(m: dict, w: str) -> dict:
    out = _heads(m, w)
    if out["vdim"] != out["dim"]:
        raise ConfigError(w + ".vdim", f"the values are the keys' projection: must equal dim ({out['dim']}), got {out['vdim']}")
    out["bias_max"] = _get(m, "bias_max", w, float)
    if out["bias_max"] <= 1:
        raise ConfigError(w + ".bias_max", f"must be greater than one, got {out['bias_max']}")
    out["bias_rows"] = _positive(m, "bias_rows", w, None)
    temp = _get(m, "q_temp", w, None, None)
    out["q_temp"] = None
    if temp is not None:
        out["q_temp"] = (_get(temp, "coef", w + ".q_temp", float), _get(temp, "every", w + ".q_temp", float))
        if out["q_temp"][1] <= 0:
            raise ConfigError(w + ".q_temp.every", f"must be greater than zero, got {out['q_temp'][1]}")
    return out


def _parallel(m: dict, w: str) -> dict:
    lf, rt, wl, wr = _get(m, "left", w), _get(m, "right", w), w + ".left", w + ".right"
    left = _heads(lf, wl)
    left["conv"] = _positive(lf, "conv", wl)
    mask = _get(lf, "mask", wl, None, None)
    left["block"] = _positive(mask, "size", wl + ".mask") if mask is not None else None
    left["rot"] = _rot(lf, wl, left["dim"])
    right = {k: _positive(rt, k, wr) for k in ("heads", "vdim", "state", "conv")}
    right["groups"], right["norm_groups"] = _positive(rt, "groups", wr, 1), _positive(rt, "norm_groups", wr, 1)
    if right["heads"] % right["groups"]:
        raise ConfigError(wr + ".groups", f"{right['groups']} does not divide {right['heads']} heads")
    if right["heads"] * right["vdim"] % right["norm_groups"]:
        raise ConfigError(wr + ".norm_groups", f"{right['norm_groups']} does not divide {right['heads'] * right['vdim']} channels")
    return {"left": left, "right": right, "left_scale": _get(m, "left_scale", w, float, 1.0), "right_scale": _get(m, "right_scale", w, float, 1.0)}


@dataclass(frozen=True)
class ZabunexConfig:
    raw: dict
    vocab: int
    width: int
    eps: float
    layers: tuple                   # dicts: type, mixer (validated), mlp

    @classmethod
    def from_dict(cls, d: dict) -> "ZabunexConfig":
        vocab = _positive(d, "vocab", "")
        width = _positive(d, "width", "")
        eps = _get(_get(d, "norm", ""), "eps", "norm", float)
        raw_layers = _get(d, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("layers", "must be a list with at least one layer")
        layers = []
        for i, L in enumerate(raw_layers):
            w = f"layers[{i}]"
            kind = _get(L, "type", w)
            if kind not in MIXERS:
                raise ConfigError(w + ".type", f"unknown layer type {kind!r}; known: {', '.join(MIXERS)}")
            mixer = (_attention if kind == "attention" else _parallel)(_get(L, "mixer", w), w + ".mixer")
            mlp = L.get("mlp")
            if mlp is not None:
                mk = _get(mlp, "kind", w + ".mlp")
                if mk != "dense":
                    raise ConfigError(w + ".mlp.kind", f"unknown feed-forward {mk!r}; known: dense")
                mlp = {"kind": mk, "ff": _positive(mlp, "ff", w + ".mlp")}
            layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
        return cls(copy.deepcopy(d), vocab, width, eps, tuple(layers))

    def to_dict(self) -> dict:
        return copy.deepcopy(self.raw)

    @property
    def stop_token_ids(self) -> tuple:
        return ()


def zabunex_plan(cfg: ZabunexConfig) -> ModelPlan:
    """Parts per layer (tensor names ``l<i>.…``); every layer runs once, in order."""
    norm = {"hidden_size": cfg.width, "eps": cfg.eps}
    heads = lambda a: {**norm, "num_heads": a["heads"], "num_kv_heads": a["kv_heads"], "head_dim": a["dim"],      # noqa: E731
                       "value_dim": a["vdim"], "scale": a["scale"], "qk_norm": "full"}
    layers = []
    for i, L in enumerate(cfg.layers):
        p, m, f = f"l{i}.", L["mixer"], L["mlp"]
        if L["type"] == "attention":
            mixer = PartSpec("window_attention", {**heads(m), "values": "keys", "query_temperature": m["q_temp"], "sink_score": 0.0,
                                                  "bias_largest": m["bias_max"], "bias_rows": m["bias_rows"]}, p + "mix.")
        else:
            lf, rt = m["left"], m["right"]
            left = PartSpec("window_attention", {**heads(lf), "conv_taps": lf["conv"], "chunk": lf["block"],
                                                 "position": PartSpec("rope", lf["rot"]) if lf["rot"] else None}, p + "mix.left.")
            right = PartSpec("state_space", {**norm, "num_heads": rt["heads"], "value_dim": rt["vdim"], "state_size": rt["state"],
                                             "groups": rt["groups"], "norm_groups": rt["norm_groups"], "conv_taps": rt["conv"]}, p + "mix.right.")
            mixer = PartSpec("parallel", {**norm, "branches": (("left", left), ("right", right)),
                                          "scales": (m["left_scale"], m["right_scale"])}, p + "mix.")
        ffn = PartSpec("dense", {"hidden_size": cfg.width, "intermediate_size": f["ff"], "activation": "relu_squared",
                                 "bias": False}, p + "mlp.") if f is not None else None
        layers.append(LayerSpec(
            arrangement="outnorm",
            norm1=PartSpec("rmsnorm", {**norm, "tensor": p + "norm1"}),
            mixer=mixer,
            norm2=PartSpec("rmsnorm", {**norm, "tensor": p + "norm2"}) if ffn is not None else None,
            ffn=ffn,
        ))
    return ModelPlan(
        embedding=PartSpec("embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tensor": "embed", "stream_rows": True}),
        layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i) for i in range(len(layers))),
        final_norm=PartSpec("rmsnorm", {**norm, "tensor": "final.norm"}),
        head=PartSpec("lm_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "tied_to": None, "tensor": "head"}),
        hidden_size=cfg.width,
        vocab_size=cfg.vocab,
        max_position=NO_POSITION_LIMIT,
        stop_token_ids=(),
    )
