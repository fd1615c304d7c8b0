"""The Ramopel decoder without a device: configuration, plan, tensor names against the naming rule, what the cache keeps
(a lender's rows reach as far back as its widest borrower sees), refusals, the plain implementation against closed
forms, and that a mistake in any mechanism would show in the test models' logits."""
import copy

import numpy as np
import pytest
import torch

import plain_ramopel as pr
from ramopel_models import CONFIGS, MIXED, ODD, WIDE, as_float64, random_config, random_weights, tensor_shapes

from camelid_b200.cache.book import KVSpec, StateSpec, flatten_specs
from camelid_b200.config.ramopel import RamopelConfig, ramopel_plan
from camelid_b200.engine.model import DecoderModel
from camelid_b200.errors import ConfigError, WeightsError
from camelid_b200.parts.recurrent import GeneralDelta


def without_free(shapes):
    """The narrow inputs' width is the stored tensors' own."""
    return {k: tuple("n" if k.endswith("mix.w1") and d == 0 or k.endswith("mix.w2") and d == 1 else n for d, n in enumerate(v))
            for k, v in shapes.items()}


@pytest.mark.parametrize("name", sorted(CONFIGS) + list(range(6)))
def test_tensor_names_follow_the_naming_rule(name):
    cfg = CONFIGS[name] if name in CONFIGS else random_config(name)
    model = DecoderModel.from_config(cfg, dtype=torch.bfloat16, device="cpu")
    got = {k: tuple(v.shape) for k, v in model.tensor_specs().items()}
    assert without_free(got) == without_free({k: v[0] for k, v in tensor_shapes(cfg).items()})


def test_plan_names_the_parts_and_their_constants():
    plan = ramopel_plan(RamopelConfig.from_dict(MIXED))
    assert [L.mixer.kind for L in plan.layers] == ["latent_attention", "general_delta"] * 3
    assert all(L.arrangement == "parallel" for L in plan.layers)
    assert [L.ffn.kind if L.ffn else None for L in plan.layers] == ["dense", "routed_experts", "routed_experts", None, None, "dense"]
    assert plan.layers[3].norm2 is None and plan.layers[0].norm2.params["tensor"] == "l0.norm2"
    assert all(L.norm1.params["offset"] == 1.0 for L in plan.layers) and plan.final_norm.params["offset"] == 1.0
    assert [e.cache_source for e in plan.schedule] == [None, None, 0, None, 0, None]
    a, b = plan.layers[0].mixer.params, plan.layers[2].mixer.params
    assert (a["window"], a["cache_window"], a["borrow_rows"], a["q_rank"]) == (9, 33, False, 24)
    assert (b["window"], b["borrow_rows"], b["q_rank"]) == (33, True, 32)
    assert a["position"].params["pairing"] == "interleaved" and a["position"].params["theta"] == 100.0
    m = plan.layers[1].ffn.params
    assert m["gate_act"] == (1.702, 0.8, 1.0) and m["shared_gate_act"] == (1.702, 0.6, 1.0) and m["router_bias"] and m["shared_output_gate"]
    assert plan.layers[2].ffn.params["shared_size"] is None and not plan.layers[2].ffn.params["shared_output_gate"]
    assert plan.layers[0].ffn.params["activation"] == "poly_norm" and plan.embedding.params["scale"] == 3.0


def test_what_the_cache_keeps():
    model = DecoderModel.from_config(MIXED, dtype=torch.bfloat16, device="cpu")
    cache = model.new_cache(256)
    # one lender with rows of 40 + 8 channels for both borrowers, as far back as the widest of the three sees
    assert cache.book.kv_specs == [KVSpec(1, 48, 33, 40, None, 0, True)] and cache.k[0].shape[0] == 1
    assert cache.entry_kv[0] == cache.entry_kv[2] == cache.entry_kv[4] == (0, 0)
    assert flatten_specs(model.blocks[1].cache_spec()) == [StateSpec((2, 24, 24), "float32", "delta")]
    # a lender that sees everything keeps everything; a layer of its own its window
    odd = DecoderModel.from_config(ODD, dtype=torch.bfloat16, device="cpu").new_cache(256)
    assert [s.window for s in odd.book.kv_specs] == [None, 64]


def test_two_matrices_side_by_side_keep_their_columns():
    model = DecoderModel.from_config(MIXED, dtype=torch.float32, device="cpu")
    w = random_weights(MIXED, 3)
    model.load_tensors(w)
    joint = model.blocks[0].w_joint
    assert torch.equal(joint, torch.cat([w["l0.mix.o"], w["l0.mlp.down"]], 1).float())
    assert model.blocks[0].mixer.w_o.data_ptr() == joint.data_ptr()          # a view: the matrices lie in memory once
    assert model.blocks[1].w_joint is None and model.blocks[3].w_joint is None
    # norm weights are kept as 1 + w in float32
    assert torch.equal(model.blocks[0].norm1.weight, w["l0.norm1"].float() + 1.0)


def test_the_narrow_input_takes_the_stored_width():
    cfg = {**MIXED, "layers": [MIXED["layers"][3]]}
    w = random_weights(cfg, 4)
    model = DecoderModel.from_config(cfg, dtype=torch.float32, device="cpu")
    model.load_tensors(w)
    assert model.blocks[0].mixer.w2.shape[1] == 8 and w["l0.mix.w1"].shape[0] == 8
    w["l0.mix.w1"], w["l0.mix.w2"] = w["l0.mix.w1"][:5].clone(), w["l0.mix.w2"][:, :5].clone()
    model.load_tensors(w)                                                    # padded with zeros to 8
    assert model.blocks[0].mixer.w2.shape[1] == 8 and float(model.blocks[0].mixer.w2[:, 5:].abs().max()) == 0.0
    w["l0.mix.w2"] = w["l0.mix.w2"][:, :4].clone()
    with pytest.raises(WeightsError):
        model.load_tensors(w)
    part = GeneralDelta({"hidden_size": 8, "num_heads": 1, "key_dim": 4}, "x.")
    assert part.decay_rate == pytest.approx(np.exp(-0.5)) and part.value_dim == 4


@pytest.mark.parametrize("path,value,key", [
    (("layers", 0, "mixer", "rot", "dims"), 6, "rot.dims"), (("layers", 0, "mixer", "rot", "base"), 0.0, "rot.base"),
    (("layers", 1, "type"), "convolution", "type"), (("layers", 0, "mlp", "kind"), "swish", "mlp.kind"),
    (("layers", 0, "mixer", "mask", "size"), 0, "mask.size"), (("vocab",), 0, "vocab"), (("layers", 0, "mixer", "q_rank"), 0, "q_rank"),
    (("layers", 1, "mlp", "router", "top"), 8, "router.top"), (("layers", 1, "mlp", "expert", "limit"), 0.0, "expert.limit"),
    (("layers", 2, "mixer", "kv_from"), 1, "kv_from"), (("layers", 2, "mixer", "kv_from"), 2, "kv_from"),
    (("layers", 4, "mixer", "kv_from"), 2, "kv_from"), (("layers", 4, "mixer", "kv_rank"), 32, "kv_rank"),
    (("layers", 2, "mixer", "rot", "base"), 50.0, "kv_from"), (("layers", 1, "mlp", "shared", "ff"), -1, "shared.ff")])
def test_refusals_name_the_key(path, value, key):
    cfg = copy.deepcopy(MIXED)
    d = cfg
    for p in path[:-1]:
        d = d[p]
    d[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        RamopelConfig.from_dict(cfg)
    assert key in str(e.value)


def test_memory_plan_counts_the_chunks_scratch():
    from camelid_b200.csrc import ops
    model = DecoderModel.from_config(WIDE, dtype=torch.bfloat16, device="cpu")
    part = model.blocks[1].mixer
    assert part.workspace_per_row() >= 4 * (5 * 128 + 128 + 2 * ops.delta_chunk_floats(64, 64) // 16)
    plan = model.memory_plan(4096, 4, 2048)
    assert plan.workspace > 2048 * part.workspace_per_row()


def test_missing_keys_take_their_defaults():
    cfg = copy.deepcopy(MIXED)
    del cfg["embedding"], cfg["layers"][0]["mixer"]["vdim"], cfg["layers"][0]["mixer"]["mask"], cfg["layers"][3]["mlp"]
    c = RamopelConfig.from_dict(cfg)
    assert c.embedding_scale == 1.0 and c.layers[0]["mixer"]["vdim"] == 16 and c.layers[0]["mixer"]["window"] is None
    assert c.layers[3]["mlp"] is None
    assert ramopel_plan(c).layers[0].mixer.params["cache_window"] == 0


def test_plain_mechanisms_against_closed_forms():
    see = pr.visible(6, 3)
    assert see[5].tolist() == [False, False, False, True, True, True] and see[1].tolist() == [True, True] + [False] * 4
    # a turn by a quarter circle of the first pair of neighbours
    x = np.array([[[1.0, 2.0, 3.0, 4.0]]])
    assert np.allclose(pr.turn_pairs(x, [np.pi / 2], 1e30)[0, 0], [-2.0, 1.0, 3.0, 4.0])
    # the delta rule by hand: one key channel; the removal rate takes from the old state, the decay acts beside it
    o = pr.delta_core(*(np.array(v) for v in ([[1.0], [2.0]], [[3.0], [1.0]], [[2.0], [5.0]], [[0.5], [0.5]], [[0.25], [0.25]])), heads=1)
    assert np.allclose(o[:, 0, 0], [6.0, 2.0 * (0.5 * 6.0 - 0.25 * 6.0 + 5.0)], rtol=1e-5)
    # two key channels: the old value of a unit key is taken away where it points, whatever the decay does
    k = np.array([[1.0, 0.0], [1.0, 0.0]])
    o = pr.delta_core(np.array([[1.0, 0.0], [1.0, 0.0]]), k, np.array([[4.0, 0.0], [7.0, 0.0]]), np.ones((2, 2)), np.ones((2, 2)), heads=1)
    assert np.allclose(o[1, 0], [7.0, 0.0], atol=1e-4)
    # normed powers of a row of equal values: every N is 1 (or the sign)
    assert np.allclose(pr.poly_norm(np.full((1, 5), -2.0), (1.0, 10.0, 100.0, 0.5), 0.0), -1.0 + 10.0 - 100.0 + 0.5)
    # the weights are the softmax over the chosen logits only, the bias counts for both
    t = {"router": np.zeros((3, 2)), "router.b": np.log(np.array([1.0, 3.0, 2.0]))}
    chosen, weights = pr.route(np.zeros((1, 2)), t, 3, 2)
    assert chosen.tolist() == [[1, 2]] and np.allclose(weights, [[0.6, 0.4]])
    # an expert beyond both limits
    y = pr.gated_expert(np.array([[9.0]]), np.array([[1.0]]), np.array([[-1.0]]), np.array([[1.0]]), 2.0)
    assert np.allclose(y, 2.0 / (1.0 + np.exp(-3.404)) * (-2.0 + 1.0))


def _other_logits(name, change, ids):
    cfg = copy.deepcopy(CONFIGS[name])
    w = as_float64(random_weights(cfg, 11))
    ref = pr.forward(cfg, w, ids)
    change(cfg, w)
    return np.abs(pr.forward(cfg, w, ids) - ref).max(axis=1)


def _set(cfg, i, key, value):
    cfg["layers"][i]["mixer"][key] = value


@pytest.mark.parametrize("name,change,first", [
    ("mixed", lambda c, w: _set(c, 0, "mask", {"size": 10}), 9), ("mixed", lambda c, w: _set(c, 2, "mask", {"size": 32}), 32),
    ("mixed", lambda c, w: _set(c, 4, "mask", {"size": 9}), 5), ("odd", lambda c, w: _set(c, 2, "mask", {"size": 71}), 70),
    ("odd", lambda c, w: _set(c, 4, "mask", {"size": 63}), 63), ("wide", lambda c, w: _set(c, 0, "mask", {"size": 131}), 130),
    ("mixed", lambda c, w: w.update({"l2.norm1": w["l2.norm1"] - 1.0}), 0), ("mixed", lambda c, w: w.update({"l1.mix.a.b": w["l1.mix.a.b"] - 30.0}), 1),
    ("mixed", lambda c, w: w.update({"l1.mix.w0": w["l1.mix.w0"] - 30.0}), 1), ("mixed", lambda c, w: w.update({"l1.mlp.router.b": 0 * w["l1.mlp.router.b"]}), 0),
    ("mixed", lambda c, w: w.update({"l1.mlp.shared.sg": w["l1.mlp.shared.sg"] * 0}), 0), ("mixed", lambda c, w: w.update({"l0.mlp.act": w["l0.mlp.act"] * [1, 1, 0, 1]}), 0),
    ("mixed", lambda c, w: c["layers"][1]["mlp"]["expert"].update({"limit": 50.0}), 0), ("mixed", lambda c, w: c["layers"][1]["mlp"]["shared"].update({"limit": 50.0}), 0)])
def test_a_mistake_in_a_mechanism_shows_in_the_logits(name, change, first):
    """The test models' weights make every mechanism count: with one planted mistake (a window one token off, norms
    without the one, no removal, no decay, no bias, half a gate, a missing power, no clamp) rows change from the first
    row on that the mechanism reaches, and no row before it."""
    ids = np.random.default_rng(5).integers(0, CONFIGS[name]["vocab"], 150)
    diff = _other_logits(name, change, ids)
    assert diff[:first].max(initial=0.0) == 0.0
    assert diff[first] > 1e-3 or first == 0
    assert np.median(diff[first:]) > 1e-2 and diff[first:].max() > 0.1


def test_benchmark_counts_every_matrix_once():
    """The bench's bytes of a decode step: with all experts reached they are the model's matrices, without the embedding
    table; the two models of the bench pass about equally many elements per token."""
    from camelid_b200 import benchmark as b
    for size in b.RAMOPEL_SIZES:
        cfg = b.ramopel_config_for(size)
        specs = DecoderModel.from_config(cfg, dtype=torch.bfloat16, device="cpu").tensor_specs()
        want = sum(int(np.prod(s.shape)) for n, s in specs.items() if len(s.shape) == 2 and n != "embed")
        got = sum(b._ramopel_matrices(L, cfg["width"], L["mlp"].get("router", {}).get("experts", 0)) for L in cfg["layers"])
        assert got + cfg["vocab"] * cfg["width"] == want
        bytes_step = b.ramopel_step_bytes(cfg, 10 ** 4, 512.0, 2)                # so many rows reach every expert
        assert abs(bytes_step["weights"] - 2 * want) < 1e-3 * want
        mine, other = b.ramopel_prefill_flops(cfg, 2048), b.kizezen_prefill_flops(b.kizezen_config_like_ramopel(size), 2048)
        assert 0.9 < mine / other < 1.1
