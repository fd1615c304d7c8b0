"""The Zabunex decoder on the device against the plain implementation (tests/plain_zabunex.py): whole prompts, decoding
through the cache and the state, portions down to two tokens, unequal batches against each sequence alone, slots and
pages used again, long decoding past every block of positions, greedy generation through the library's entry point, the trace
runner, and the kernels of each mechanism alone with inputs made so that one distance, a far key, a lost tap or a
lost state shows."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zabunex as pz
from zabunex_models import CONFIGS, as_float64, random_config, write_model
import helpers
from helpers import assert_same_engine, tokens

pytestmark = pytest.mark.gpu

SEEDS = {"mixed": 41, "odd": 42, "wide": 43}
LENGTHS = {"mixed": 150, "odd": 171, "wide": 330}
# bfloat16: a state carried over hundreds of tokens and norms of its read-outs in parts pass rounding on, which a dense
# decoder does not; single rows get a wider bound than the library's, the mean error a tight one
BF16_ROW, BF16_MEAN = 8e-2, 6e-3


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        d = str(tmp_path_factory.mktemp("zabunex_" + name))
        out[name] = (d, as_float64(write_model(d, cfg, SEEDS[name])))
    return out


_models: dict = {}
_plain: dict = {}


def model(folders, name, dtype):
    import camelid_b200
    if (name, dtype) not in _models:
        _models[(name, dtype)] = camelid_b200.load(folders[name][0], dtype=dtype)
    return _models[(name, dtype)]


def plain(folders, name, ids):
    key = (name, tuple(ids))
    if key not in _plain:
        _plain[key] = torch.from_numpy(pz.forward(CONFIGS[name], folders[name][1], list(ids)))
    return _plain[key]


def assert_close(got, ref, dtype, what=""):
    if dtype == "float32":
        return helpers.assert_close(got, ref, dtype, what)
    got = torch.as_tensor(got)
    rows = helpers.row_errors(got, ref)
    assert float(rows.max()) <= BF16_ROW, f"{what}: row {int(rows.argmax())} is off by {float(rows.max()):.3e} of its largest logit"
    assert float(rows.median()) <= helpers.TOL[dtype], f"{what}: the median row is off by {float(rows.median()):.3e}"
    m = helpers.mean_err(got, ref)
    assert m <= BF16_MEAN, f"{what}: mean error {m:.3e}"


def run_cut(lm, cache, ids, cut):
    """Feed ``ids`` in portions of the sizes ``cut`` (the rest one by one); logits of every position."""
    from camelid_b200.engine.model import StepEntry
    slot = cache.alloc_slot()
    out, at = [], 0
    for n in list(cut) + [1] * (len(ids) - sum(cut)):
        out.append(lm.step(cache, [StepEntry(slot, ids[at:at + n], list(range(n)))]).cpu())
        at += n
    cache.free_slot(slot)
    return torch.cat(out)


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("odd", "float32"), ("wide", "float32"), ("wide", "bfloat16")])
def test_whole_prompt_and_decoding_match_plain(cuda, folders, name, dtype):
    lm = model(folders, name, dtype)
    ids = tokens(SEEDS[name], LENGTHS[name], CONFIGS[name]["vocab"])
    ref = plain(folders, name, ids)
    cache = lm.new_cache(1024)
    whole = run_cut(lm, cache, ids, [len(ids)])
    assert_close(whole, ref, dtype, f"{name} whole prompt")
    decoded = run_cut(lm, cache, ids, [len(ids) - 40])         # the last tokens one by one (captured steps)
    assert_close(decoded, ref, dtype, f"{name} decoded")
    if dtype == "float32":
        assert_same_engine(whole, decoded, f"{name} whole against decoded", tol=5e-5)
    lm.model.check_device_errors()
    cache.book.audit()


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_sizes_no_tensor_core_product_takes_in_bfloat16(cuda, folders, name):
    """bfloat16 on the CUDA-core fallbacks, whole, in portions and decoded."""
    lm = model(folders, name, "bfloat16")
    ids = tokens(SEEDS[name], 90, CONFIGS[name]["vocab"])
    got = run_cut(lm, lm.new_cache(256), ids, [60, 2])
    assert_close(got, plain(folders, name, ids), "bfloat16", f"{name} in bfloat16")


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(cuda, tmp_path, seed):
    """Sizes, head counts, the order of the layers, blocks, taps, groups, feed-forwards and constants drawn from a
    seed: a whole prompt, the same tokens with the last 30 decoded one by one, and two sequences in one batch."""
    import camelid_b200
    from camelid_b200.engine.model import StepEntry
    cfg = random_config(seed)
    weights = as_float64(write_model(str(tmp_path), cfg, 50 + seed))
    lm = camelid_b200.load(str(tmp_path), dtype="float32")
    ids, short = tokens(seed, 160, cfg["vocab"]), tokens(90 + seed, 21, cfg["vocab"])
    ref, ref_short = torch.from_numpy(pz.forward(cfg, weights, ids)), torch.from_numpy(pz.forward(cfg, weights, short))
    cache = lm.new_cache(512)
    assert_close(run_cut(lm, cache, ids, [len(ids)]), ref, "float32", f"seed {seed} whole prompt")
    assert_close(run_cut(lm, cache, ids, [len(ids) - 30]), ref, "float32", f"seed {seed} decoded")
    a, b = cache.alloc_slot(), cache.alloc_slot()
    both = lm.step(cache, [StepEntry(a, short[:20], list(range(20))), StepEntry(b, ids[:150], list(range(150)))]).cpu()
    one = lm.step(cache, [StepEntry(a, short[20:], [0]), StepEntry(b, ids[150:151], [0])]).cpu()
    assert_close(torch.cat([both[:20], one[:1]]), ref_short, "float32", f"seed {seed} the short sequence of a batch")
    assert_close(torch.cat([both[20:], one[1:]]), ref[:151], "float32", f"seed {seed} the long sequence of a batch")
    cache.free_slot(a)
    cache.free_slot(b)
    cache.book.audit()
    lm.model.check_device_errors()


@pytest.mark.parametrize("seed", range(6))
def test_configurations_for_the_tensor_core_kernels_in_bfloat16(cuda, tmp_path, seed):
    """Drawn configurations whose heads and states the bfloat16 tensor-core kernels take: whole prompts, portions,
    decoding and a batch, against the plain implementation at the bounds of bfloat16."""
    import camelid_b200
    from camelid_b200.engine.model import StepEntry
    cfg = random_config(seed, tensor_cores=True)
    weights = as_float64(write_model(str(tmp_path), cfg, 70 + seed))
    lm = camelid_b200.load(str(tmp_path), dtype="bfloat16")
    ids, short = tokens(seed, 300, cfg["vocab"]), tokens(90 + seed, 21, cfg["vocab"])
    ref, ref_short = torch.from_numpy(pz.forward(cfg, weights, ids)), torch.from_numpy(pz.forward(cfg, weights, short))
    cache = lm.new_cache(1024)
    assert_close(run_cut(lm, cache, ids, [len(ids)]), ref, "bfloat16", f"seed {seed} whole prompt")
    assert_close(run_cut(lm, cache, ids, [130, 2, 138]), ref, "bfloat16", f"seed {seed} portions and decoding")
    a, b = cache.alloc_slot(), cache.alloc_slot()
    both = lm.step(cache, [StepEntry(a, short[:20], list(range(20))), StepEntry(b, ids[:290], list(range(290)))]).cpu()
    one = lm.step(cache, [StepEntry(a, short[20:], [0]), StepEntry(b, ids[290:291], [0])]).cpu()
    assert_close(torch.cat([both[:20], one[:1]]), ref_short, "bfloat16", f"seed {seed} the short sequence of a batch")
    assert_close(torch.cat([both[20:], one[1:]]), ref[:291], "bfloat16", f"seed {seed} the long sequence of a batch")
    cache.free_slot(a)
    cache.free_slot(b)
    lm.model.check_device_errors()


def test_every_token_decoded_alone(cuda, folders):
    """From the first token on: the first tokens of a sequence, taps and blocks as they fill."""
    for name in ("mixed", "odd"):
        lm = model(folders, name, "float32")
        ids = tokens(7, 100, CONFIGS[name]["vocab"])
        got = run_cut(lm, lm.new_cache(256), ids, [])
        assert_close(got, plain(folders, name, ids), "float32", f"{name} token by token")


@pytest.mark.parametrize("name,cut", [("mixed", [7, 2, 3, 2, 50, 1, 1, 2, 64, 2]), ("odd", [64, 2, 63, 1, 2, 5]),
                                      ("wide", [2, 126, 2, 3, 128, 2, 60]), ("odd", [1, 2, 2, 3, 70, 71]), ("mixed", [16, 17, 15, 33, 31])])
def test_portions_of_a_prompt(cuda, folders, name, cut):
    lm = model(folders, name, "float32")
    ids = tokens(SEEDS[name], LENGTHS[name], CONFIGS[name]["vocab"])
    got = run_cut(lm, lm.new_cache(1024), ids, cut)
    assert_close(got, plain(folders, name, ids), "float32", f"{name} in portions {cut}")


def test_portions_in_bfloat16_on_the_tensor_core_attention(cuda, folders):
    lm = model(folders, "wide", "bfloat16")
    ids = tokens(SEEDS["wide"], LENGTHS["wide"], CONFIGS["wide"]["vocab"])
    got = run_cut(lm, lm.new_cache(1024), ids, [150, 2, 70, 100])
    assert_close(got, plain(folders, "wide", ids), "bfloat16", "wide in portions")


@pytest.mark.parametrize("name,dtype", [("mixed", "float32"), ("odd", "float32"), ("wide", "float32"), ("wide", "bfloat16")])
def test_unequal_batch_against_each_alone(cuda, folders, name, dtype):
    """Prompts of 1, 17 and 135 tokens start together, are decoded together and end one after the other."""
    from camelid_b200.engine.model import StepEntry
    lm = model(folders, name, dtype)
    vocab = CONFIGS[name]["vocab"]
    seqs = [tokens(100 + i, n, vocab) for i, n in enumerate((9, 30, 150))]
    prompt = [1, 17, 135]
    cache = lm.new_cache(1024)
    slots = [cache.alloc_slot() for _ in seqs]
    got = [[] for _ in seqs]
    logits = lm.step(cache, [StepEntry(s, q[:p], list(range(p))) for s, q, p in zip(slots, seqs, prompt)]).cpu()
    at = 0
    for i, p in enumerate(prompt):
        got[i].append(logits[at:at + p])
        at += p
    done, live = list(prompt), [0, 1, 2]
    while live:
        logits = lm.step(cache, [StepEntry(slots[i], [seqs[i][done[i]]], [0]) for i in live]).cpu()
        for j, i in enumerate(live):
            got[i].append(logits[j:j + 1])
            done[i] += 1
        for i in [i for i in live if done[i] == len(seqs[i])]:
            cache.free_slot(slots[i])
        live = [i for i in live if done[i] < len(seqs[i])]
    for i, q in enumerate(seqs):
        assert_close(torch.cat(got[i]), plain(folders, name, q), dtype, f"{name} sequence {i} of a batch")
    cache.book.audit()


def test_slots_and_pages_used_again(cuda, folders):
    """A cache of four pages and one slot: every sequence gets the slot, the state and the pages the one before gave
    back; layers with blocks of positions give old pages back on the way."""
    for name in ("mixed", "odd"):
        lm = model(folders, name, "float32")
        cache = lm.new_cache(256, max_slots=1)
        for i, n in enumerate((200, 75, 250)):
            ids = tokens(200 + i, n, CONFIGS[name]["vocab"])
            got = run_cut(lm, cache, ids, [n - 10])
            assert_close(got, plain(folders, name, ids), "float32", f"{name}: sequence {i} in a slot used before")
            cache.book.audit()
        assert cache.book.slots.n_free == 1 and all(p.n_free == p.n for p in cache.book.pools)


def test_long_decoding_past_every_block(cuda, folders):
    lm = model(folders, "mixed", "float32")
    ids = tokens(5, 300, CONFIGS["mixed"]["vocab"])
    got = run_cut(lm, lm.new_cache(512), ids, [3])
    assert_close(got, plain(folders, "mixed", ids), "float32", "297 tokens decoded one by one")
    lm = model(folders, "wide", "float32")
    ids = tokens(6, 300, CONFIGS["wide"]["vocab"])
    got = run_cut(lm, lm.new_cache(512), ids, [120])
    assert_close(got, plain(folders, "wide", ids), "float32", "180 tokens decoded past blocks of 130 and 200")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(cuda, folders, dtype):
    """``generate`` (scheduler, batches, the decode loop on the device) picks the plain implementation's tokens."""
    lm = model(folders, "wide", dtype)
    cfg = CONFIGS["wide"]
    prompts = [tokens(300, 5, cfg["vocab"]), tokens(301, 19, cfg["vocab"]), tokens(302, 1, cfg["vocab"])]
    for _ in range(2):                                         # the second call uses the slots again
        out = lm.generate(prompts, max_tokens=12)
        for p, new in zip(prompts, out):
            assert len(new) == 12
            seq = list(p)
            for tok in new:
                ref = plain(folders, "wide", seq)
                top2 = torch.topk(ref[-1], 2).values
                if dtype == "float32" or float(top2[0] - top2[1]) > 0.5:
                    assert tok == int(ref[-1].argmax()), (seq, new)
                seq.append(tok)


def test_weights_drawn_on_the_device_match_the_folder(cuda, tmp_path):
    import camelid_b200
    from camelid_b200.weights.random_init import write_random_model
    cfg = CONFIGS["mixed"]
    folder = write_random_model(str(tmp_path / "m"), cfg, seed=5)
    a = camelid_b200.load(folder, dtype="bfloat16")
    b = camelid_b200.from_random(cfg, seed=5, dtype="bfloat16")
    prompts = [tokens(1, 12, cfg["vocab"]), tokens(2, 3, cfg["vocab"])]
    assert a.generate(prompts, max_tokens=6) == b.generate(prompts, max_tokens=6)


def test_trace_runner_replays_a_zabunex_model(cuda, folders, tmp_path):
    folder, _ = folders["odd"]
    cfg = CONFIGS["odd"]
    a, b = tokens(1, 40, cfg["vocab"]), tokens(2, 4, cfg["vocab"])
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:38], "want": [0, 32, 33, 37]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[38:39], "want": []}, {"id": "b", "tokens": b[1:2], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[39:40], "want": [0]}, {"id": "b", "tokens": b[2:3], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[3:4], "want": [0]}], "end": ["b"]}]
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    r = subprocess.run([sys.executable, exe, "--model", folder, "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "128"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    ra, rb = plain(folders, "odd", a), plain(folders, "odd", b)
    want = {0: torch.stack([ra[0], ra[32], ra[33], ra[37], rb[0]]), 1: rb[1:2], 2: torch.stack([ra[39], rb[2]]), 3: rb[3:4]}
    for i, ref in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]))
        helpers.assert_close(got, ref, "float32", f"step {i}")


# ---- each mechanism's kernels alone -------------------------------------------------------------

def arrays(cuda, starts, news, slots=None):
    """The packed-row arrays of a step."""
    dev = lambda a: torch.as_tensor(np.asarray(a), dtype=torch.int32, device=cuda)      # noqa: E731
    row0 = np.concatenate([[0], np.cumsum(news)[:-1]])
    return {"row_seq": dev(np.repeat(np.arange(len(news)), news)),
            "row_pos": dev(np.concatenate([np.arange(s, s + n) for s, n in zip(starts, news)])),
            "seq_row0": dev(row0), "seq_new": dev(news), "seq_start": dev(starts),
            "seq_slot": dev(slots if slots is not None else np.arange(len(news)))}


def portions(n, cut):
    at = 0
    for s in list(cut) + [1] * (n - sum(cut)):
        yield at, s
        at += s




@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,Dv,taps,rot,splits", [(4, 2, 8, 12, 4, 4, 1), (3, 1, 7, 5, 2, 0, 1), (2, 2, 64, 64, 5, 64, 1), (6, 3, 16, 8, 1, 8, 1),
                                                      (4, 4, 32, 32, 4, 16, 3), (5, 5, 6, 9, 8, 2, 2)])
def test_short_convolution_before_the_norms(cuda, H, G, D, Dv, taps, rot, splits, dtype):
    """Two sequences in slots that held other inputs, fed in portions down to one token: what the preparing kernel writes is the
    plain convolution, norm and rotation of the whole sequences."""
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(taps)
    cols, n, eps = H * D + G * (D + Dv), [70, 24], 1e-5
    u = [torch.randn(k, cols, generator=gen) for k in n]
    w, qw, kw = torch.randn(cols, taps, generator=gen), 1.0 + 0.3 * torch.randn(H * D, generator=gen), 1.0 + 0.3 * torch.randn(G * D, generator=gen)
    freq = torch.tensor([100.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)] or [0.0])
    state = torch.randn(4, max(taps - 1, 1), cols, generator=gen).to(cuda)
    slots = [2, 0]
    table = torch.tensor([[0, 1], [2, 3]], dtype=torch.int32, device=cuda)
    k_pages, v_pages = torch.zeros(4, G, 64, D, dtype=dtype, device=cuda), torch.zeros(4, G, 64, Dv, dtype=dtype, device=cuda)
    q_rows = [[], []]
    at = [0, 0]
    steps = [(5, 1), (2, 2), (1, 1), (1, 1), (40, 3)] + [(1, 1)] * 3 + [(18, 13)]
    for new in steps:
        a = arrays(cuda, at, list(new), slots)
        rows = torch.cat([u[i][at[i]:at[i] + new[i]] for i in (0, 1)])
        parts = torch.randn(splits, *rows.shape, generator=gen)
        parts[0] = rows - parts[1:].sum(0)
        proj = parts.to(cuda)
        q = torch.empty(rows.shape[0], H * D, dtype=dtype, device=cuda)
        decode = max(new) == 1
        ops.qkv_prepare(proj, qw.to(cuda), kw.to(cuda), 2, eps, freq.to(cuda), rot, False, a["row_seq"], a["row_pos"], table, q, k_pages, v_pages,
                        H, G, D, Dv, conv=(w.t().contiguous().to(cuda), state, a["seq_row0"], a["seq_slot"], decode))
        if taps > 1 and not decode:
            ops.keep_last_rows(rows.to(cuda).contiguous(), 0, cols, state, a["seq_row0"], a["seq_new"], a["seq_start"], a["seq_slot"], 2)
        q = q.float().cpu()
        q_rows[0].append(q[:new[0]])
        q_rows[1].append(q[new[0]:])
        at = [at[i] + new[i] for i in (0, 1)]
    assert at == n
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for i in (0, 1):
        m = at[i]
        x = pz.short_conv(u[i][:m].double().numpy(), w.double().numpy())
        pos = np.arange(m)
        rq = pz.turn_halves(pz.rms_norm(x[:, :H * D], qw.double().numpy(), eps).reshape(m, H, D), pos, rot, 100.0).reshape(m, -1)
        rk = pz.turn_halves(pz.rms_norm(x[:, H * D:H * D + G * D], kw.double().numpy(), eps).reshape(m, G, D), pos, rot, 100.0)
        rv = x[:, H * D + G * D:].reshape(m, G, Dv)
        pages = table[i].long()
        gk = k_pages[pages].permute(0, 2, 1, 3).reshape(128, G, D)[:m].double().cpu().numpy()
        gv = v_pages[pages].permute(0, 2, 1, 3).reshape(128, G, Dv)[:m].double().cpu().numpy()
        for got, ref in ((torch.cat(q_rows[i]).double().numpy(), rq), (gk, rk), (gv, rv)):
            assert np.abs(got - ref).max() <= tol * max(1.0, np.abs(ref).max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,D,coef,every", [(4, 2, 8, 0.3, 10), (3, 3, 7, 0.7, 1), (2, 1, 64, 0.2, 64), (5, 5, 6, 0.0, 1), (2, 2, 33, 0.5, 2.5)])
def test_values_from_the_keys_and_queries_that_grow(cuda, H, G, D, coef, every, dtype):
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(D)
    n, start, eps = 100, 25, 1e-5
    proj = torch.randn(n, H * D + G * D, generator=gen)
    qw, kw = 1.0 + 0.3 * torch.randn(H * D, generator=gen), 1.0 + 0.3 * torch.randn(G * D, generator=gen)
    a = arrays(cuda, [start], [n])
    table = torch.tensor([[1, 0]], dtype=torch.int32, device=cuda)
    k_pages, v_pages = torch.zeros(2, G, 64, D, dtype=dtype, device=cuda), torch.zeros(2, G, 64, D, dtype=dtype, device=cuda)
    q = torch.empty(n, H * D, dtype=dtype, device=cuda)
    ops.qkv_prepare(proj.to(cuda), qw.to(cuda), kw.to(cuda), 2, eps, torch.zeros(1, device=cuda), 0, False, a["row_seq"], a["row_pos"], table, q,
                    k_pages, v_pages, H, G, D, D, share_values=True, temperature=(coef, every) if coef else None)
    x = proj.double().numpy()
    rq = pz.rms_norm(x[:, :H * D], qw.double().numpy(), eps) * pz.temperature(np.arange(start, start + n), coef, every)[:, None]
    rk = pz.rms_norm(x[:, H * D:], kw.double().numpy(), eps)
    at = lambda pages: pages[[1, 0]].permute(0, 2, 1, 3).reshape(128, -1)[start:start + n].double().cpu().numpy()      # noqa: E731
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    for got, ref in ((q.double().cpu().numpy(), rq), (at(k_pages), rk), (at(v_pages), x[:, H * D:])):
        assert np.abs(got - ref).max() <= tol * np.abs(ref).max()


def paged(cuda, k, v, dtype, order):
    """k, v [n, G, D | Dv] in pages handed out in the given order; everything else in the pool holds large numbers."""
    n, G = k.shape[:2]
    kp = torch.full((len(order) + 1, G, 64, k.shape[2]), 50.0, dtype=dtype, device=cuda)
    vp = torch.full((len(order) + 1, G, 64, v.shape[2]), 50.0, dtype=dtype, device=cuda)
    for b, page in enumerate(order):
        for src, dst in ((k, kp), (v, vp)):
            piece = src[b * 64:(b + 1) * 64]
            dst[page, :, :piece.shape[0]] = piece.permute(1, 0, 2).to(dtype).to(cuda)
    return kp, vp, torch.tensor([order], dtype=torch.int32, device=cuda)


@pytest.mark.parametrize("H,G,D,n_rel,loved", [(6, 2, 64, 100, 37), (4, 4, 128, 300, 64), (3, 1, 64, 65, 64), (2, 2, 128, 17, 0), (16, 2, 64, 130, 129), (6, 6, 128, 2, 1)])
def test_bias_by_distance_and_the_extra_term(cuda, H, G, D, n_rel, loved):
    """A bias that stands out at one distance: every query finds the value that far back (and, where the table's last number
    stands out, all values at least that far back), in prompts on either kernel, in a portion that starts mid-sequence and alone;
    and ordinary tables against the plain softmax."""
    from camelid_b200.csrc import ops
    from camelid_b200.parts import linear
    gen = torch.Generator().manual_seed(n_rel)
    n, scale = 330, 0.1
    q, k = torch.randn(n, H, D, generator=gen), torch.randn(n, G, D, generator=gen)
    v = torch.randn(n, G, D, generator=gen)
    for spike in (False, True):
        rel = torch.randn(H, n_rel, generator=gen) * (0.0 if spike else 1.5)
        if spike:
            rel[:, loved] = 25.0
        by = np.minimum(np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0), n_rel - 1)
        for dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 2e-2)):
            qd, kd, vd = (t.to(dtype).double().numpy() for t in (q, k, v))
            ref = pz.attend(qd, kd, vd, scale, pz.causal(n), rel.double().numpy()[:, by], 1.0).reshape(n, -1)
            kp, vp, table = paged(cuda, k, v, dtype, [3, 0, 5, 1, 2, 4])
            sink, bias = torch.zeros(H, device=cuda), rel.to(cuda)
            qr = q.to(dtype).reshape(n, -1).to(cuda).contiguous()
            for start in (0, 201, n - 1):
                a = arrays(cuda, [start], [n - start])
                wide = torch.zeros(n - start, H * D + 16, dtype=dtype, device=cuda)
                out = wide[:, 8:8 + H * D]                           # rows of another stride
                ops.window_attention(qr[start:].contiguous(), kp, vp, table, a["row_seq"], a["row_pos"], None, None, None, 0, out, H, G, D, D, 0,
                                     scale, 0, sink, distance_bias=bias, out_scale=0.5)
                assert np.abs(2.0 * out.double().cpu().numpy() - ref[start:]).max() <= tol * np.abs(ref).max(), (spike, dtype, start)
                assert float(wide[:, :8].abs().max()) == 0.0 and float(wide[:, -8:].abs().max()) == 0.0
                if dtype != torch.bfloat16 or start == n - 1:
                    continue
                rows, hpc, chunks = ops.attn_tc_tiling(H, G)
                q0 = list(range(0, n - start, rows))
                tiles = [torch.tensor(t, dtype=torch.int32, device=cuda) for t in ([0] * len(q0), q0)]
                wide.zero_()
                err = linear._err_word(out.device)
                ops.attn_prefill_tc(qr[start:].contiguous(), out, kp, vp, table, tiles[0], tiles[1], len(q0), a["seq_row0"], a["seq_start"], a["seq_new"],
                                    H, G, D, rows, hpc, chunks, 0, scale, err, sink=sink, raw_bias=(rel.double() / scale).float().to(cuda), out_scale=0.5)
                got = 2.0 * out.double().cpu().numpy()
                assert np.abs(got - ref[start:]).max() <= tol * np.abs(ref).max(), (spike, "tensor cores", start)
                assert float(wide[:, :8].abs().max()) == 0.0 and float(wide[:, -8:].abs().max()) == 0.0
                linear.check_errors()


def test_the_extra_term_takes_its_share(cuda):
    """One key with score ln 3: its weight is 3 / 4."""
    from camelid_b200.csrc import ops
    q = torch.full((1, 16), np.log(3.0) / 16, device=cuda)
    kp, vp = torch.ones(1, 1, 64, 16, device=cuda), torch.full((1, 1, 64, 16), 2.0, device=cuda)
    out = torch.empty(1, 16, device=cuda)
    a = arrays(cuda, [0], [1])
    ops.window_attention(q, kp, vp, torch.zeros(1, 1, dtype=torch.int32, device=cuda), a["row_seq"], a["row_pos"], None, None, None, 0, out, 1, 1, 16, 16,
                         0, 1.0, 0, torch.zeros(1, device=cuda))
    assert torch.allclose(out, torch.full_like(out, 1.5))


SSM_CUTS = {"whole": [], "portions": [64, 2, 63, 1, 1, 2, 17], "alone": [1] * 40 + [100]}


def ssm_arrays(cuda, seed, n, H, G, N, P):
    """Random inputs of the recurrence: decays that keep something for hundreds of tokens in some heads, a few in others."""
    gen = torch.Generator().manual_seed(seed)
    x, B, C = torch.randn(n, H, P, generator=gen), torch.randn(n, G, N, generator=gen), torch.randn(n, G, N, generator=gen)
    dt = torch.nn.functional.softplus(torch.randn(n, H, generator=gen) - 1.0)
    A_log = torch.linspace(-5.0, 1.5, H) if H > 1 else torch.tensor([-4.0])
    D = torch.randn(H, generator=gen)
    return x, B, C, dt, A_log, D


def run_chunks(cuda, rows, gates, d, a_log, state, a, y, new, H, G, N, P):
    """The chunked kernels on the packed rows of a step."""
    from camelid_b200.csrc import ops
    seqs, q0 = [], []
    for i, m in enumerate(new):
        starts = list(range(0, m, ops.SSM_CHUNK))
        seqs += [i] * len(starts)
        q0 += starts
    t = [torch.tensor(v, dtype=torch.int32, device=cuda) for v in (seqs, q0)]
    scores = torch.full((len(seqs), G, ops.SSM_CHUNK, ops.SSM_CHUNK), float("nan"), device=cuda)
    prev = torch.full((len(seqs), H, P, N), float("nan"), device=cuda)
    steps = torch.full((len(seqs), H, 3, ops.SSM_CHUNK), float("nan"), device=cuda)
    ops.ssm_chunks(rows, (0, H * P, H * P + G * N), gates, a_log, d, t[0], t[1], len(seqs), a["seq_row0"], a["seq_new"], a["seq_start"], a["seq_slot"],
                   state, scores, steps, prev, y, len(new), H, G, N, P)


def run_scan(cuda, data, cut, slot, state, G, chunked):
    """One sequence through the recurrence's kernels in portions; [n, H * P]. ``chunked``: portions of many tokens run by chunks."""
    from camelid_b200.csrc import ops
    x, B, C, dt, A_log, D = data
    n, H, P = x.shape
    N = B.shape[2]
    rows = torch.cat([x.reshape(n, -1), B.reshape(n, -1), C.reshape(n, -1)], 1).to(cuda)
    gates = torch.cat([dt, torch.exp(-torch.exp(A_log) * dt)], 1).to(cuda)
    d, a_log = D.to(cuda), A_log.to(cuda)
    out = []
    cut = list(cut) or [n]
    for at, m in portions(n, cut):
        a = arrays(cuda, [at], [m], [slot])
        y = torch.empty(m, H * P, device=cuda)
        part, g = rows[at:at + m].contiguous(), gates[at:at + m].contiguous()
        if chunked and m > 1:
            run_chunks(cuda, part, g, d, a_log, state, a, y, [m], H, G, N, P)
        else:
            ops.ssm_scan(part, (0, H * P, H * P + G * N), g, d, state, a["seq_row0"], a["seq_new"], a["seq_start"], a["seq_slot"], y, 1, H, G, N, P)
        out.append(y.cpu())
    return torch.cat(out).double().numpy()


@pytest.mark.parametrize("H,G,N,P", [(4, 2, 16, 8), (6, 2, 44, 36), (3, 1, 128, 64), (2, 2, 7, 5), (1, 1, 256, 20), (8, 1, 33, 16), (5, 5, 3, 40)])
@pytest.mark.parametrize("cut", sorted(SSM_CUTS))
def test_the_recurrence_token_by_token(cuda, H, G, N, P, cut):
    data = ssm_arrays(cuda, N + P, 200, H, G, N, P)
    ref = pz.state_space(*(t.double().numpy() for t in data)).reshape(200, -1)
    state = torch.randn(3, H, P, N, device=cuda)                    # what the slot's last sequence left
    got = run_scan(cuda, data, SSM_CUTS[cut], 1, state, G, False)
    assert np.abs(got - ref).max() <= 2e-5 * np.abs(ref).max()


@pytest.mark.parametrize("H,G,N,P", [(4, 2, 16, 8), (6, 2, 44, 36), (3, 1, 128, 64), (2, 2, 4, 4), (1, 1, 256, 20), (8, 1, 36, 16), (5, 5, 40, 140), (2, 1, 96, 128)])
@pytest.mark.parametrize("cut", sorted(SSM_CUTS))
def test_the_recurrence_by_chunks(cuda, H, G, N, P, cut):
    """Whole chunks, ragged ones, portions that continue a state, and single tokens in between."""
    data = ssm_arrays(cuda, N + P, 200, H, G, N, P)
    ref = pz.state_space(*(t.double().numpy() for t in data)).reshape(200, -1)
    state = torch.randn(3, H, P, N, device=cuda)
    got = run_scan(cuda, data, SSM_CUTS[cut], 1, state, G, True)
    assert np.abs(got - ref).max() <= 2e-5 * np.abs(ref).max()
    token_by_token = torch.zeros(3, H, P, N, device=cuda)           # the same state is left behind
    run_scan(cuda, data, [], 1, token_by_token, G, False)
    assert float((state[1] - token_by_token[1]).abs().max()) <= 2e-5 * float(token_by_token[1].abs().max())


def test_several_sequences_by_chunks(cuda):
    """Sequences of 1, 130, 64 and 63 tokens in one step, slots out of order."""
    H, G, N, P = 4, 2, 32, 16
    news, slots = [1, 130, 64, 63], [3, 0, 4, 1]
    all_data = [ssm_arrays(cuda, i, m, H, G, N, P)[:4] + ssm_arrays(cuda, 0, 1, H, G, N, P)[4:] for i, m in enumerate(news)]
    rows = torch.cat([torch.cat([x.reshape(m, -1), B.reshape(m, -1), C.reshape(m, -1)], 1) for (x, B, C, _, _, _), m in zip(all_data, news)]).to(cuda)
    A_log, D = all_data[0][4:]
    dt = torch.cat([d[3] for d in all_data])
    gates = torch.cat([dt, torch.exp(-torch.exp(A_log) * dt)], 1).to(cuda)
    state, y = torch.randn(5, H, P, N, device=cuda), torch.empty(sum(news), H * P, device=cuda)
    untouched = state[2].clone()
    run_chunks(cuda, rows, gates, D.to(cuda), A_log.to(cuda), state, arrays(cuda, [0] * 4, news, slots), y, news, H, G, N, P)
    ref = np.concatenate([pz.state_space(*(t.double().numpy() for t in d)).reshape(m, -1) for d, m in zip(all_data, news)])
    assert np.abs(y.double().cpu().numpy() - ref).max() <= 2e-5 * np.abs(ref).max()
    assert torch.equal(state[2], untouched)


def test_decays_that_leave_nothing(cuda):
    """Steps so large that a chunk's decay is zero in 32 bits: no overflow, the last token's share alone."""
    H, G, N, P, n = 2, 1, 8, 4, 130
    x, B, C, dt, A_log, D = ssm_arrays(cuda, 5, n, H, G, N, P)
    data = (x, B, C, dt * 20.0, torch.tensor([2.5, 0.5]), D)
    ref = pz.state_space(*(t.double().numpy() for t in data)).reshape(n, -1)
    for chunked in (False, True):
        got = run_scan(cuda, data, [], 0, torch.zeros(1, H, P, N, device=cuda), G, chunked)
        assert np.abs(got - ref).max() <= 2e-5 * np.abs(ref).max()


def test_a_far_key_stays_in_the_state(cuda):
    """A token whose B alone points along one channel, written at position 3 and asked for at 200 and more by C along it."""
    H, G, N, P, n = 2, 1, 24, 8, 260
    x, B, C, dt, A_log, D = ssm_arrays(cuda, 1, n, H, G, N, P)
    B[:, :, 5], C[:, :, 5], D = 0.0, 0.0, D * 0
    B[3, 0], C[200:, 0] = 0.0, 0.0
    B[3, 0, 5], C[200:, 0, 5] = 4.0, 2.0
    A_log = torch.tensor([-8.0, -6.0])
    data = (x, B, C, dt, A_log, D)
    ref = pz.state_space(*(t.double().numpy() for t in data)).reshape(n, -1)
    assert np.abs(ref[200:]).max() > 0.5
    state = torch.zeros(1, H, P, N, device=cuda)
    for cut in ([], [150, 2, 3, 90], [4] + [1] * 60):
        for chunked in (False, True):
            got = run_scan(cuda, data, cut, 0, state, G, chunked)
            assert np.abs(got[200:] - ref[200:]).max() <= 2e-5 * np.abs(ref[200:]).max()


@pytest.mark.parametrize("inner,channels,heads,taps,splits", [(32, 48, 4, 4, 1), (21, 34, 3, 2, 1), (64, 128, 8, 6, 1), (16, 24, 2, 1, 1), (40, 56, 5, 4, 5), (7, 9, 1, 3, 2)])
def test_inputs_of_the_recurrence(cuda, inner, channels, heads, taps, splits):
    """Convolution with bias and SiLU, steps and decays, through portions and single tokens of two sequences in slots that held
    other inputs."""
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(taps)
    width = inner + channels + heads
    u = [torch.randn(60, width, generator=gen), torch.randn(40, width, generator=gen)]
    w, b = torch.randn(channels, taps, generator=gen), torch.randn(channels, generator=gen)
    dt_b, a_log = torch.randn(heads, generator=gen), torch.randn(heads, generator=gen)
    state = torch.randn(3, max(taps - 1, 1), channels, generator=gen).to(cuda)
    dev = [t.to(cuda) for t in (w.t().contiguous(), b, dt_b, a_log)]
    got = [[], []]
    at = [0, 0]
    for new in [(1, 1), (2, 9), (1, 1), (1, 1), (20, 2), (1, 1), (30, 20)]:
        a = arrays(cuda, at, list(new), [2, 1])
        rows = torch.cat([u[i][at[i]:at[i] + new[i]] for i in (0, 1)])
        parts = torch.randn(splits, *rows.shape, generator=gen)
        parts[0] = rows - parts[1:].sum(0)
        decode = max(new) == 1
        out, gates, z = (torch.empty(rows.shape[0], k, device=cuda) for k in (channels, 2 * heads, inner))
        ops.ssm_inputs(parts.to(cuda), *dev, state, a["row_seq"], a["row_pos"], a["seq_row0"], a["seq_slot"], out, gates, inner, z, update_state=decode)
        if taps > 1 and not decode:
            ops.keep_last_rows(rows.to(cuda).contiguous(), inner, channels, state, a["seq_row0"], a["seq_new"], a["seq_start"], a["seq_slot"], 2)
        all_cols = torch.cat([z, out, gates], 1).double().cpu().numpy()
        got[0].append(all_cols[:new[0]])
        got[1].append(all_cols[new[0]:])
        at = [at[i] + new[i] for i in (0, 1)]
    for i in (0, 1):
        x = u[i][:at[i]].double().numpy()
        conv = pz.silu(pz.short_conv(x[:, inner:inner + channels], w.double().numpy(), b.double().numpy()))
        dt = pz.softplus(x[:, inner + channels:] + dt_b.double().numpy())
        ref = np.concatenate([x[:, :inner], conv, dt, np.exp(-np.exp(a_log.double().numpy()) * dt)], 1)
        assert np.abs(np.concatenate(got[i]) - ref).max() <= 3e-5


@pytest.mark.parametrize("rows,width,groups", [(5, 64, 1), (300, 96, 3), (2, 33, 11), (7, 4096, 8), (3, 2050, 2), (1, 16384, 1)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gate_before_the_norm_in_parts(cuda, rows, width, groups, dtype):
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(width)
    y, z, w = torch.randn(rows, width, generator=gen), torch.randn(rows, width + 12, generator=gen), 1.0 + 0.3 * torch.randn(width, generator=gen)
    y[:, :width // groups] *= 30.0                                   # a part of another size than the others
    wide = torch.zeros(rows, width + 8, dtype=dtype, device=cuda)
    ops.gated_group_norm(y.to(cuda), z.to(cuda)[:, 4:4 + width], w.to(cuda), groups, 1e-5, wide[:, :width])
    ref = pz.gated_group_norm(y.double().numpy(), z[:, 4:4 + width].double().numpy(), w.double().numpy(), groups, 1e-5)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert np.abs(wide[:, :width].double().cpu().numpy() - ref).max() <= tol * np.abs(ref).max()
    assert float(wide[:, width:].abs().max()) == 0.0
