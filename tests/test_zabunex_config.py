"""The Zabunex decoder without a device: configuration, plan, tensor names against the naming rule, what the cache keeps,
refusals, the plain implementation against closed forms, and that a mistake in any mechanism would show in the test
models' logits."""
import copy

import numpy as np
import pytest
import torch

import plain_zabunex as pz
from zabunex_models import CONFIGS, MIXED, ODD, as_float64, random_config, random_weights, tensor_shapes

from camelid_b200.cache.book import KVSpec, StateSpec, flatten_specs
from camelid_b200.config.zabunex import ZabunexConfig, zabunex_plan
from camelid_b200.engine.model import DecoderModel
from camelid_b200.errors import ConfigError, WeightsError
from camelid_b200.parts.position import rotary_frequencies
from camelid_b200.parts.window_attention import WindowAttention, distance_buckets


@pytest.mark.parametrize("name", sorted(CONFIGS) + list(range(6)))
def test_tensor_names_follow_the_naming_rule(name):
    cfg = CONFIGS[name] if name in CONFIGS else random_config(name)
    got = {k: tuple(v.shape) for k, v in DecoderModel.from_config(cfg, dtype=torch.bfloat16, device="cpu").tensor_specs().items()}
    want = {k: v[0] for k, v in tensor_shapes(cfg).items()}
    # the rows of a bias table are the stored tensor's own
    free = lambda d: {k: ("rows",) + v[1:] if k.endswith(".rel") else v for k, v in d.items()}      # noqa: E731
    assert free(got) == free(want)


def test_plan_names_the_parts_and_their_constants():
    plan = zabunex_plan(ZabunexConfig.from_dict(MIXED))
    assert [L.mixer.kind for L in plan.layers] == ["parallel", "window_attention", "window_attention", "parallel", "parallel", "window_attention"]
    assert all(L.arrangement == "outnorm" and L.norm1.params["tensor"] == f"l{i}.norm1" for i, L in enumerate(plan.layers))
    assert [L.ffn.params["intermediate_size"] if L.ffn else None for L in plan.layers] == [72, 104, None, None, 88, 56]
    assert plan.layers[2].norm2 is None and plan.layers[0].ffn.params["activation"] == "relu_squared" and not plan.layers[0].ffn.params["bias"]
    p = plan.layers[0].mixer.params
    assert p["scales"] == (0.7, 1.3)
    (_, a), (_, b) = p["branches"]
    assert (a.kind, a.prefix, a.params["conv_taps"], a.params["chunk"], a.params["value_dim"]) == ("window_attention", "l0.mix.left.", 3, 33, 12)
    rot = a.params["position"].params
    assert (rot["rotary_dim"], rot["theta"], rot["pairing"], rot["scaling"]["factor"]) == (8, 100.0, "split", 2.0)
    assert (b.kind, b.params["state_size"], b.params["groups"], b.params["norm_groups"], b.params["conv_taps"]) == ("state_space", 10, 2, 4, 4)
    m = plan.layers[1].mixer.params
    assert m["values"] == "keys" and m["query_temperature"] == (0.4, 25.0) and m["sink_score"] == 0.0 and m["bias_largest"] == 90.0
    assert plan.layers[2].mixer.params["query_temperature"] is None and m["qk_norm"] == "full"
    assert plan.layers[3].mixer.params["branches"][0][1].params["position"] is None


def test_what_the_cache_keeps():
    model = DecoderModel.from_config(MIXED, dtype=torch.bfloat16, device="cpu")
    cache = model.new_cache(256)
    assert KVSpec(2, 16, None, 12, 33) in cache.book.kv_specs and KVSpec(2, 20) in cache.book.kv_specs
    assert flatten_specs(model.blocks[0].cache_spec())[1:] == [
        StateSpec((2, 6 * 16 + 2 * (16 + 12)), "float32", "qkv_conv"), StateSpec((4, 8, 10), "float32", "ssm"), StateSpec((3, 32 + 40), "float32", "ssm_conv")]
    # one tap: nothing of the convolution is carried (a row that nobody reads keeps the shape)
    odd = DecoderModel.from_config(ODD, dtype=torch.bfloat16, device="cpu")
    assert [s.shape for s in flatten_specs(odd.blocks[2].cache_spec()) if getattr(s, "name", "") == "ssm_conv"] == [(1, 45 + 12)]


def test_weights_side_by_side():
    model = DecoderModel.from_config(MIXED, dtype=torch.float32, device="cpu")
    w = random_weights(MIXED, 3)
    model.load_tensors(w)
    mix = model.blocks[0].mixer
    assert torch.equal(mix.w_joint, torch.cat([w["l0.mix.left.o"], w["l0.mix.right.o"]], 1).float())
    assert mix.branches[0].w_o.data_ptr() == mix.w_joint.data_ptr()          # a view: the matrices lie in memory once
    # every branch's rows of the stacked input matrix start on a multiple of 8, the rows between are zero
    (a0, an), (b0, bn) = mix.in_cols
    assert a0 == 0 and b0 % 8 == 0 and torch.equal(mix.w_in[b0:b0 + 32 + 72 + 4], w["l0.mix.right.in"].float())
    assert mix.w_in.shape[0] % 8 == 0 and float(mix.w_in[b0 + 108:].abs().max()) == 0.0
    # a branch's scale goes into its rows: the attention's factor, the state-space half's norm weight
    assert mix.branches[0].out_scale == 0.7
    assert torch.allclose(mix.branches[1].norm_w, w["l0.mix.right.norm"].float() * 1.3)
    model.load_tensors(w)                                                    # (loading again starts from the stored weights)
    assert mix.branches[0].out_scale == 0.7 and torch.allclose(mix.branches[1].norm_w, w["l0.mix.right.norm"].float() * 1.3)
    assert torch.equal(mix.branches[1].conv_w, w["l0.mix.right.conv"].float().t())
    assert torch.equal(model.blocks[1].mixer.sink_w, torch.zeros(4))


@pytest.mark.parametrize("rows,largest", [(32, 250), (4, 17), (6, 200.5), (2, 9), (10, 300), (30, 16), (7, 50)])
def test_the_bias_table_written_out_by_distance(rows, largest):
    table = distance_buckets(rows, largest)
    assert table == [pz.bucket(d, rows, largest) for d in range(len(table))]
    assert table[-1] == rows - 1 and all(pz.bucket(d, rows, largest) == rows - 1 for d in range(len(table), len(table) + 500))
    assert table[:rows // 2] == list(range(rows // 2)) and sorted(table) == table
    part = WindowAttention({"hidden_size": 8, "num_heads": 2, "num_kv_heads": 1, "head_dim": 4, "qk_norm": "full", "bias_largest": largest,
                            "scale": 0.5}, "x.")
    rel = torch.randn(rows, 2, generator=torch.Generator().manual_seed(1))
    part._load_distance_bias(rel, "cpu")
    assert torch.equal(part.rel, rel[table].t()) and torch.allclose(part.raw_rel, part.rel / 0.5)


def test_a_bias_table_that_does_not_fit_is_refused():
    w = random_weights(MIXED, 4)
    model = DecoderModel.from_config(MIXED, dtype=torch.float32, device="cpu")
    w["l2.mix.rel"] = torch.zeros(44, 3, dtype=torch.bfloat16)               # half of the rows reach beyond the bias's 20 positions
    with pytest.raises(WeightsError):
        model.load_tensors(w)
    w["l2.mix.rel"] = torch.zeros(1, 3, dtype=torch.bfloat16)
    with pytest.raises(WeightsError):
        model.load_tensors(w)


@pytest.mark.parametrize("path,value,key", [
    (("layers", 1, "type"), "convolution", "type"), (("layers", 0, "mlp", "kind"), "moe", "mlp.kind"), (("vocab",), 0, "vocab"),
    (("layers", 1, "mixer", "vdim"), 24, "vdim"), (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"), (("layers", 1, "mixer", "bias_max"), 1, "bias_max"),
    (("layers", 1, "mixer", "q_temp", "every"), 0, "q_temp.every"), (("layers", 0, "mixer", "left", "mask", "size"), 0, "mask.size"),
    (("layers", 0, "mixer", "left", "conv"), 0, "left.conv"), (("layers", 0, "mixer", "left", "rot", "dims"), 18, "rot.dims"),
    (("layers", 0, "mixer", "left", "rot", "scaling", "factor"), 0, "scaling.factor"), (("layers", 0, "mixer", "right", "groups"), 3, "right.groups"),
    (("layers", 0, "mixer", "right", "norm_groups"), 5, "norm_groups"), (("layers", 0, "mixer", "right", "state"), -1, "right.state")])
def test_refusals_name_the_key(path, value, key):
    cfg = copy.deepcopy(MIXED)
    d = cfg
    for p in path[:-1]:
        d = d[p]
    d[path[-1]] = value
    with pytest.raises(ConfigError) as e:
        ZabunexConfig.from_dict(cfg)
    assert key in str(e.value)


def test_options_of_the_parts_that_exclude_each_other():
    base = {"hidden_size": 8, "num_heads": 2, "num_kv_heads": 1, "head_dim": 4}
    for more in ({"values": "keys", "value_dim": 6}, {"bias_largest": 1.0}, {"sink": True, "sink_score": 0.0}, {"conv_taps": 0},
                 {"conv_taps": 3, "bias": True}, {"difference": 0.5, "values": "keys"}, {"query_temperature": (0.1, 0)}):
        with pytest.raises(ConfigError):
            WindowAttention({**base, **more}, "x.")


def test_missing_keys_take_their_defaults():
    cfg = copy.deepcopy(MIXED)
    m, a = cfg["layers"][0]["mixer"], cfg["layers"][1]["mixer"]
    del m["left"]["vdim"], m["left"]["mask"], m["left"]["rot"]["scaling"], m["left_scale"], m["right"]["groups"], a["kv_heads"], a["q_temp"]
    c = ZabunexConfig.from_dict(cfg)
    L = c.layers[0]["mixer"]
    assert L["left"]["vdim"] == 16 and L["left"]["block"] is None and L["left"]["rot"]["scaling"]["factor"] == 1.0
    assert L["left_scale"] == 1.0 and L["right"]["groups"] == 1 and c.layers[1]["mixer"]["kv_heads"] == 4 and c.layers[1]["mixer"]["q_temp"] is None


def test_linear_scaling_divides_every_frequency():
    f = rotary_frequencies(16, 500.0, {"rope_type": "linear", "factor": 4.0})
    assert np.allclose(f, 500.0 ** (-np.arange(8) / 8.0) / 4.0, rtol=1e-7)


def test_plain_mechanisms_against_closed_forms():
    # a convolution by hand: zeros before the start, the last tap the token's own
    y = pz.short_conv(np.array([[1.0], [2.0], [3.0]]), np.array([[10.0, 1.0]]), np.array([0.5]))
    assert np.allclose(y[:, 0], [1.5, 12.5, 23.5])
    # a turn of the first pair of halves by a quarter circle (halved by the factor 2 from a half circle)
    t = pz.turn_halves(np.array([[[1.0, 2.0, 3.0, 4.0, 9.0]]]), [np.pi], 4, 1e30, 2.0)
    assert np.allclose(t[0, 0], [-3.0, 2.0, 1.0, 4.0, 9.0])
    see = pz.same_block(5, 2)
    assert see[2].tolist() == [False, False, True, False, False] and see[3].tolist() == [False, False, True, True, False]
    # equal scores of ln 2: each weight 2 / (1 + 2 n); without the extra term 1 / n
    q, k, v = np.ones((3, 1, 1)), np.full((3, 1, 1), np.log(2.0)), np.ones((3, 1, 1))
    assert np.allclose(pz.attend(q, k, v, 1.0, pz.causal(3), None, 1.0)[:, 0, 0], [2 / 3, 4 / 5, 6 / 7])
    assert np.allclose(pz.attend(q, k, v, 1.0, pz.causal(3))[:, 0, 0], 1.0)
    assert np.allclose(pz.temperature([0, 8, 9, 28], 2.0, 10), 1.0 + 2.0 * np.log([1.0, 1.0, 2.0, 3.0]))
    assert [pz.bucket(n, 8, 64) for n in (0, 3, 4, 7, 8, 15, 16, 31, 32, 64, 1000)] == [0, 3, 4, 4, 5, 5, 6, 6, 7, 7, 7]
    # the recurrence by hand: a half-life of one step, two heads that share B and C
    y = pz.state_space(np.array([[[1.0], [10.0]], [[2.0], [20.0]]]), np.full((2, 1, 1), 3.0), np.full((2, 1, 1), 0.5), np.full((2, 2), 2.0),
                       np.log(np.full(2, np.log(2.0) / 2.0)), np.array([0.0, 1.0]))
    assert np.allclose(y[:, :, 0], [[3.0, 30.0 + 10.0], [1.5 + 6.0, 15.0 + 60.0 + 20.0]])
    g = pz.gated_group_norm(np.array([[3.0, 4.0, 0.0, 5.0]]), np.full((1, 4), 50.0), np.ones(4), 2, 0.0)
    assert np.allclose(g, np.array([[3.0, 4.0, 0.0, 5.0]]) / np.sqrt(12.5))


def _other_logits(name, change, ids):
    cfg = copy.deepcopy(CONFIGS[name])
    w = as_float64(random_weights(cfg, 11))
    ref = pz.forward(cfg, w, ids)
    change(cfg, w)
    return np.abs(pz.forward(cfg, w, ids) - ref).max(axis=1)


def _set(c, path, value):
    for p in path[:-1]:
        c = c[p]
    c[path[-1]] = value


def _one_tap_less(w, name):
    w[name] = w[name].copy()
    w[name][:, 0] = 0.0


@pytest.mark.parametrize("name,change,first", [
    ("mixed", lambda c, w: _set(c, ("layers", 0, "mixer", "left", "mask", "size"), 34), 33),
    ("mixed", lambda c, w: _set(c, ("layers", 3, "mixer", "left", "mask", "size"), 8), 8),
    ("odd", lambda c, w: _set(c, ("layers", 1, "mixer", "left", "mask", "size"), 65), 64),
    ("wide", lambda c, w: _set(c, ("layers", 0, "mixer", "left", "mask", "size"), 131), 130),
    ("mixed", lambda c, w: _set(c, ("layers", 1, "mixer", "q_temp", "every"), 26), 24),
    ("mixed", lambda c, w: _set(c, ("layers", 1, "mixer", "q_temp"), None), 24),
    ("mixed", lambda c, w: _set(c, ("layers", 1, "mixer", "bias_max"), 70), 0),
    ("mixed", lambda c, w: w.update({"l1.mix.rel": w["l1.mix.rel"] * 0}), 0),
    ("mixed", lambda c, w: w.update({"l2.mix.rel": np.concatenate([w["l2.mix.rel"][:-1], w["l2.mix.rel"][:1]])}), 0),
    ("mixed", lambda c, w: _one_tap_less(w, "l0.mix.left.q.conv"), 2), ("mixed", lambda c, w: _one_tap_less(w, "l0.mix.left.k.conv"), 2),
    ("mixed", lambda c, w: _one_tap_less(w, "l0.mix.left.v.conv"), 2), ("mixed", lambda c, w: _one_tap_less(w, "l0.mix.right.conv"), 3),
    ("mixed", lambda c, w: w.update({"l0.mix.right.conv.b": w["l0.mix.right.conv.b"] * 0}), 0),
    ("mixed", lambda c, w: w.update({"l0.mix.right.dt_bias": w["l0.mix.right.dt_bias"] + 0.5}), 0),
    ("mixed", lambda c, w: w.update({"l0.mix.right.A_log": w["l0.mix.right.A_log"] + 1.0}), 1),
    ("mixed", lambda c, w: w.update({"l0.mix.right.D": w["l0.mix.right.D"] * 0}), 0),
    ("mixed", lambda c, w: _set(c, ("layers", 0, "mixer", "right", "norm_groups"), 1), 0),
    ("mixed", lambda c, w: _set(c, ("layers", 0, "mixer", "left_scale"), 1.3), 0),
    ("mixed", lambda c, w: _set(c, ("layers", 0, "mixer", "left", "rot", "scaling"), None), 1),
    ("wide", lambda c, w: _set(c, ("layers", 0, "mixer", "left", "rot", "dims"), 64), 1)])
def test_a_mistake_in_a_mechanism_shows_in_the_logits(name, change, first):
    """The test models' weights make every mechanism count: with one planted mistake rows change from the first row on that
    the mechanism reaches, and no row before it."""
    ids = np.random.default_rng(5).integers(0, CONFIGS[name]["vocab"], 150)
    diff = _other_logits(name, change, ids)
    assert diff[:first].max(initial=0.0) == 0.0
    assert np.median(diff[first:]) > 1e-2 and diff[first:].max() > 5e-2


def test_no_extra_term_or_values_from_normed_keys_would_show(monkeypatch):
    ids = np.random.default_rng(6).integers(0, MIXED["vocab"], 80)
    w = as_float64(random_weights(MIXED, 11))
    ref = pz.forward(MIXED, w, ids)
    real = pz.attend
    monkeypatch.setattr(pz, "attend", lambda q, k, v, scale, see, bias=None, extra=0.0: real(q, k, v, scale, see, bias, 0.0))
    assert np.median(np.abs(pz.forward(MIXED, w, ids) - ref).max(axis=1)) > 1e-2
    monkeypatch.setattr(pz, "attend", lambda q, k, v, scale, see, bias=None, extra=0.0: real(q, k, k if extra else v, scale, see, bias, extra))
    assert np.median(np.abs(pz.forward(MIXED, w, ids) - ref).max(axis=1)) > 1e-2


def test_benchmark_counts_every_matrix_once():
    """The bench's bytes of a decode step count the model's matrices without the embedding table; the two models of the bench pass
    about equally many elements per token."""
    from camelid_b200 import benchmark as b
    for size in b.ZABUNEX_SIZES:
        cfg, other = b.zabunex_config_for(size), b.kizezen_config_like_zabunex(size)
        specs = DecoderModel.from_config(cfg, dtype=torch.bfloat16, device="cpu").tensor_specs()
        want = sum(int(np.prod(s.shape)) for n, s in specs.items() if len(s.shape) == 2 and n != "embed" and not n.endswith((".conv", ".rel")))
        bytes_step = b.zabunex_step_bytes(cfg, 8, 512.0, 2)
        assert bytes_step["weights"] == 2 * want
        assert 0.98 < bytes_step["weights"] / b.kizezen_step_bytes(other, 8, 512.0, 2)["weights"] < 1.02
        assert 0.9 < b.zabunex_prefill_flops(cfg, 2048) / b.kizezen_prefill_flops(other, 2048) < 1.1


def test_memory_plan_counts_states_and_the_chunks_scratch():
    from zabunex_models import WIDE
    model = DecoderModel.from_config(WIDE, dtype=torch.bfloat16, device="cpu")
    part = model.blocks[0].mixer.branches[1]
    assert part.workspace_per_row() >= 4 * (part.in_width + 2 * 64 + 4 * 32 * 64 // 64)
    plan, more = model.memory_plan(4096, 4, 2048), model.memory_plan(4096, 5, 2048)
    assert model.blocks[0].mixer.workspace_per_row() == part.workspace_per_row()             # through the mixers side by side
    assert plan.workspace > 2048 * part.workspace_per_row()
    states = 4 * 32 * 64 + 3 * (128 + 256) + 2 * 64 * 128 + 3 * (128 + 256)          # S and the kept inputs of both parallel layers' right sides
    kept = 3 * (384 + 128 + 256) + 2 * (384 + 128 + 64)                              # and of their left sides
    assert more.cache - plan.cache == 4 * (states + kept)
