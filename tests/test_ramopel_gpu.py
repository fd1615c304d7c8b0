"""The Ramopel decoder on the device against the plain implementation (tests/plain_ramopel.py): whole prompts, decoding
through the cache and the state, portions down to two tokens, unequal batches against each sequence alone, slots and
pages used again, long decoding past every window, greedy generation through the library's entry point, the trace
runner, and the kernels of each mechanism alone with inputs made so that a window's edge, a far key or a lost state
shows."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_ramopel as pr
from ramopel_models import CONFIGS, as_float64, random_config, write_model
import helpers
from helpers import assert_same_engine, tokens

pytestmark = pytest.mark.gpu

SEEDS = {"mixed": 41, "odd": 42, "wide": 43}
LENGTHS = {"mixed": 150, "odd": 171, "wide": 330}
# bfloat16: a state carried over hundreds of tokens and per-head norms of its read-outs pass rounding on, which a dense
# decoder does not; single rows get a wider bound than the library's, the mean error a tight one
BF16_ROW, BF16_MEAN = 8e-2, 6e-3


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        d = str(tmp_path_factory.mktemp("ramopel_" + name))
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
        _plain[key] = torch.from_numpy(pr.forward(CONFIGS[name], folders[name][1], list(ids)))
    return _plain[key]


def steady_rows(cfg, weights, ids, floor=0.02, gap=0.1):
    """Rows that bfloat16 can be held to: no read-out of the delta rule that is just what cancellation left (the norm behind
    it keeps only its direction), no choice of experts that rounding could turn."""
    cond, gaps = [], []
    pr.forward(cfg, weights, list(ids), conditioning=cond, gaps=gaps)
    ok = np.ones(len(ids), bool)
    for c in cond:
        ok &= c > floor
    for g in gaps:
        ok &= g > gap
    return ok


def assert_close(got, ref, dtype, what="", rows_ok=None):
    if dtype == "float32":
        return helpers.assert_close(got, ref, dtype, what)
    got = torch.as_tensor(got)
    if rows_ok is not None and not rows_ok.all():
        assert rows_ok.mean() > 0.6, f"{what}: too few steady rows for a test"
        keep = torch.from_numpy(np.nonzero(rows_ok)[0])
        got, ref = got[keep], ref[keep]
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
    ok = steady_rows(CONFIGS[name], folders[name][1], ids) if dtype == "bfloat16" else None
    cache = lm.new_cache(1024)
    whole = run_cut(lm, cache, ids, [len(ids)])
    assert_close(whole, ref, dtype, f"{name} whole prompt", ok)
    decoded = run_cut(lm, cache, ids, [len(ids) - 40])         # the last tokens one by one (captured steps)
    assert_close(decoded, ref, dtype, f"{name} decoded", ok)
    if dtype == "float32":
        assert_same_engine(whole, decoded, f"{name} whole against decoded", tol=5e-5)
    lm.model.check_device_errors()
    cache.book.audit()


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_sizes_no_tensor_core_product_takes_in_bfloat16(cuda, folders, name):
    """bfloat16 on the CUDA-core fallbacks; routed layers choose, so only rows without a close call are compared, and the
    tokens before them that chose otherwise leave a trace: the median row is held to the library's bound."""
    lm = model(folders, name, "bfloat16")
    ids = tokens(SEEDS[name], 60, CONFIGS[name]["vocab"])
    ref = plain(folders, name, ids)
    ok = torch.from_numpy(np.nonzero(steady_rows(CONFIGS[name], folders[name][1], ids, gap=0.05))[0])
    got = run_cut(lm, lm.new_cache(256), ids, [40, 2])
    rows = helpers.row_errors(got[ok], ref[ok])
    assert len(ok) > 20 and float(rows.median()) <= 3e-2 and float(rows.quantile(0.9)) <= 0.15


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(cuda, tmp_path, seed):
    """Sizes, head counts, the order of the layers, windows, borrowed rows, feed-forwards and constants drawn from a
    seed: a whole prompt, the same tokens with the last 30 decoded one by one, and two sequences in one batch."""
    import camelid_b200
    from camelid_b200.engine.model import StepEntry
    cfg = random_config(seed)
    weights = as_float64(write_model(str(tmp_path), cfg, 50 + seed))
    lm = camelid_b200.load(str(tmp_path), dtype="float32")
    ids, short = tokens(seed, 160, cfg["vocab"]), tokens(90 + seed, 21, cfg["vocab"])
    ref, ref_short = torch.from_numpy(pr.forward(cfg, weights, ids)), torch.from_numpy(pr.forward(cfg, weights, short))
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
    """Drawn configurations whose widths and latents the bfloat16 tensor-core kernels take: whole prompts, portions,
    decoding and a batch, against the plain implementation at the bounds of bfloat16."""
    import camelid_b200
    from camelid_b200.engine.model import StepEntry
    cfg = random_config(seed, tensor_cores=True)
    weights = as_float64(write_model(str(tmp_path), cfg, 70 + seed))
    lm = camelid_b200.load(str(tmp_path), dtype="bfloat16")
    ids, short = tokens(seed, 300, cfg["vocab"]), tokens(90 + seed, 21, cfg["vocab"])
    ref, ref_short = torch.from_numpy(pr.forward(cfg, weights, ids)), torch.from_numpy(pr.forward(cfg, weights, short))
    ok, ok_short = steady_rows(cfg, weights, ids), steady_rows(cfg, weights, short)
    cache = lm.new_cache(1024)
    assert_close(run_cut(lm, cache, ids, [len(ids)]), ref, "bfloat16", f"seed {seed} whole prompt", ok)
    assert_close(run_cut(lm, cache, ids, [130, 2, 138]), ref, "bfloat16", f"seed {seed} portions and decoding", ok)
    a, b = cache.alloc_slot(), cache.alloc_slot()
    both = lm.step(cache, [StepEntry(a, short[:20], list(range(20))), StepEntry(b, ids[:290], list(range(290)))]).cpu()
    one = lm.step(cache, [StepEntry(a, short[20:], [0]), StepEntry(b, ids[290:291], [0])]).cpu()
    assert_close(torch.cat([both[:20], one[:1]]), ref_short, "bfloat16", f"seed {seed} the short sequence of a batch", ok_short)
    assert_close(torch.cat([both[20:], one[1:]]), ref[:291], "bfloat16", f"seed {seed} the long sequence of a batch", ok[:291])
    cache.free_slot(a)
    cache.free_slot(b)
    lm.model.check_device_errors()


def test_every_token_decoded_alone(cuda, folders):
    """From the first token on: the first tokens of a sequence and the windows as they fill."""
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
    assert_close(got, plain(folders, "wide", ids), "bfloat16", "wide in portions", steady_rows(CONFIGS["wide"], folders["wide"][1], ids))


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
        ok = steady_rows(CONFIGS[name], folders[name][1], q) if dtype == "bfloat16" else None
        assert_close(torch.cat(got[i]), plain(folders, name, q), dtype, f"{name} sequence {i} of a batch", ok)
    cache.book.audit()


def test_slots_and_pages_used_again(cuda, folders):
    """A cache of four pages and one slot: every sequence gets the slot, the state and the pages the one before gave
    back; windowed layers give old pages back on the way."""
    for name in ("mixed", "odd"):
        lm = model(folders, name, "float32")
        cache = lm.new_cache(256, max_slots=1)
        for i, n in enumerate((200, 75, 250)):
            ids = tokens(200 + i, n, CONFIGS[name]["vocab"])
            got = run_cut(lm, cache, ids, [n - 10])
            assert_close(got, plain(folders, name, ids), "float32", f"{name}: sequence {i} in a slot used before")
            cache.book.audit()
        assert cache.book.slots.n_free == 1 and all(p.n_free == p.n for p in cache.book.pools)


def test_long_decoding_past_every_window(cuda, folders):
    lm = model(folders, "mixed", "float32")
    ids = tokens(5, 300, CONFIGS["mixed"]["vocab"])
    got = run_cut(lm, lm.new_cache(512), ids, [3])
    assert_close(got, plain(folders, "mixed", ids), "float32", "297 tokens decoded one by one")
    lm = model(folders, "wide", "float32")
    ids = tokens(6, 300, CONFIGS["wide"]["vocab"])
    got = run_cut(lm, lm.new_cache(512), ids, [120])
    assert_close(got, plain(folders, "wide", ids), "float32", "180 tokens decoded past windows of 130, 200 and 64")


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


def test_trace_runner_replays_a_ramopel_model(cuda, folders, tmp_path):
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


@pytest.mark.parametrize("rows,hidden,splits", [(3, 64, 4), (70, 130, 3), (200, 256, 0), (5, 2048, 9), (300, 44, 0), (2, 37, 2), (9, 70, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_two_norms_of_the_same_rows_in_one_pass(cuda, rows, hidden, splits, dtype):
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(1)
    x = torch.randn(rows, hidden, generator=gen) * 3
    part = torch.randn(max(splits, 1), rows, hidden, generator=gen)
    w1, w2 = 1 + 0.3 * torch.randn(hidden, generator=gen), 1 + 0.3 * torch.randn(hidden, generator=gen)
    full = (x + part.sum(0) if splits else x).double().numpy()
    xd = x.to(cuda).clone()
    a, b = torch.empty(rows, hidden, dtype=dtype, device=cuda), torch.empty(rows, hidden, dtype=dtype, device=cuda)
    ops.rmsnorm(xd, w1.to(cuda), 1e-5, a, None, part.to(cuda) if splits else None, w2.to(cuda), b)
    tol = 1e-5 if dtype == torch.float32 else 2e-2
    for got, w in ((a, w1), (b, w2)):
        ref = torch.from_numpy(pr.rms_norm(full, w.double().numpy(), 1e-5))
        assert float((got.cpu().double() - ref).abs().max()) < tol * float(ref.abs().max())
    assert float((xd.cpu().double() - torch.from_numpy(full)).abs().max()) < 1e-4


@pytest.mark.parametrize("rows,width,splits,pad", [(1, 72, 3, 0), (9, 4096, 9, 16), (40, 137, 1, 5), (300, 256, 0, 8), (130, 100, 0, 4), (7, 37, 0, 3),
                                                   (2, 14336, 2, 0)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_weighted_sum_of_normed_powers(cuda, rows, width, splits, pad, dtype):
    """From split sums, and in place on rows of the compute type; into rows that lie inside wider ones."""
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(2)
    coef = torch.tensor([0.7, -1.3, 0.4, 0.25])
    part = torch.randn(max(splits, 1), rows, width, generator=gen) * 1.5
    if splits == 0:
        part = part.to(dtype).float()
    ref = torch.from_numpy(pr.poly_norm(part.sum(0).double().numpy(), coef.double().numpy(), 1e-5))
    wide = torch.full((rows, width + pad), 9.0, dtype=dtype, device=cuda)
    out = wide[:, pad:]
    if splits == 0:
        out.copy_(part[0])
    ops.poly_norm(part.to(cuda) if splits else out, coef.to(cuda), 1e-5, out)
    tol = 2e-5 if dtype == torch.float32 else 1e-2
    assert float((out.cpu().double() - ref).abs().max()) < tol * float(ref.abs().max())
    assert pad == 0 or float((wide[:, :pad].float() - 9.0).abs().max()) == 0.0


def _latent_case(T, m, window, dtype, seed=3):
    """Projections' rows in which some positions' latents are asked for by every query: at the window's edge as seen from
    later rows, at page borders and far back. Returns them with the plain result."""
    gen = torch.Generator().manual_seed(seed)
    H, D, R, Dv, C, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
    t = {"uk": torch.randn(H * D, C, generator=gen) / C ** 0.5, "uv": torch.randn(H * Dv, C, generator=gen) / C ** 0.5,
         "uq": torch.randn(H * (D + R), Q, generator=gen) / Q ** 0.5, "dkv.norm": 1 + 0.3 * torch.randn(C, generator=gen),
         "dq.norm": 1 + 0.3 * torch.randn(Q, generator=gen)}
    t = {n: (x.to(torch.bfloat16) if x.dim() == 2 else x).double() for n, x in t.items()}
    qlat, down = torch.randn(T, Q, generator=gen), torch.randn(T, C + R, generator=gen)
    loved = sorted({0, 1, 62, 63, 64, 65, 127, 128, T - window - 1, T - window, T - window + 1} & set(range(T)))
    direction = torch.randn(C, generator=gen)
    for j in loved:
        down[j, :C] = direction * (3.0 + 0.1 * j) + torch.randn(C, generator=gen) * 0.3
    # every query points at the loved latents' keys: the query latent's common part maps onto uk . direction
    want = (t["uk"] @ (direction.double() / direction.norm() * C ** 0.5)).view(H, D)
    want = torch.cat([want, torch.zeros(H, R, dtype=torch.float64)], 1).reshape(-1)
    common = torch.linalg.lstsq(t["uq"], want).solution
    qlat = qlat * 0.3 + common.float() / common.norm().float() * Q ** 0.5
    tn = {n: x.numpy() for n, x in t.items()}
    eps = 1e-5
    cq = pr.rms_norm(qlat.double().numpy(), tn["dq.norm"], eps)
    rows = pr.latent_rows(down.double().numpy(), tn, m, eps)
    ref = pr.latent_core(cq @ tn["uq"].T, *rows, tn, m)
    return qlat, down, t, torch.from_numpy(ref), eps


@pytest.mark.parametrize("dtype,C,R,tol", [(torch.float32, 40, 8, 5e-5), (torch.bfloat16, 36, 6, 5e-2), (torch.bfloat16, 64, 16, 5e-2)])
@pytest.mark.parametrize("window", [1, 5, 33, 64, 65, 100, 200, None])
@pytest.mark.parametrize("cut", [[330], [100, 2, 60, 130, 2]])
def test_window_over_latent_rows(cuda, cut, window, dtype, C, R, tol):
    """A position that every query asks for is seen while it is inside the window and not a row longer. Whole prompts,
    portions and single tokens, pages in another order than positions; the rows of pages that left the window are
    overwritten with numbers that would show."""
    from camelid_b200.csrc import ops
    T = 330
    m = {"heads": 5, "dim": 12, "rot_dim": R, "vdim": 20, "kv_rank": C, "q_rank": 24, "scale": 0.5, "rot": {"base": 50.0, "dims": R}}
    if window:
        m["mask"] = {"size": window}
    qlat, down, t, ref, eps = _latent_case(T, m, window or 0, dtype)
    if window and window < 200:
        wider = pr.latent_core(pr.rms_norm(qlat.double().numpy(), t["dq.norm"].numpy(), eps) @ t["uq"].numpy().T,
                               *pr.latent_rows(down.double().numpy(), {n: x.numpy() for n, x in t.items()}, m, eps),
                               {n: x.numpy() for n, x in t.items()}, {**m, "mask": {"size": window + 1}})
        assert float(np.abs(wider[window:] - ref.numpy()[window:]).max()) > 0.2      # one position more would show
    H, D, Dv, Q = m["heads"], m["dim"], m["vdim"], m["q_rank"]
    pages = (T + 63) // 64
    order = list(range(pages))[::-1]
    kp = torch.zeros(pages, 1, 64, C + R, dtype=dtype, device=cuda)
    inv_freq = torch.tensor([50.0 ** (-2.0 * i / R) for i in range(R // 2)], dtype=torch.float32, device=cuda)
    uk_t = t["uk"].view(H, D, C).transpose(1, 2).contiguous().to(cuda, dtype)
    uv = t["uv"].view(H, Dv, C).contiguous().to(cuda, dtype)
    first_proj = torch.cat([qlat, down], 1).to(cuda)
    got = []
    for at, n in portions(T, cut):
        a = arrays(cuda, [at], [n])
        row = list(order)
        if window:                                     # what a windowed cache has given back by now
            for b in range(max(0, at - window + 1) // 64):
                kp[order[b]] = 100.0
                row[b] = -1
        table = torch.tensor([row + [-1]], dtype=torch.int32, device=cuda)
        cq = torch.empty(n, Q, device=cuda, dtype=dtype)
        common = (eps, inv_freq, True, 1.0, a["row_seq"], a["row_pos"], table)
        ops.latent_prepare(first_proj[at:at + n], t["dkv.norm"].float().to(cuda), *common, None, None, kp, 0, D, R, C, None, cq,
                           t["dq.norm"].float().to(cuda))
        q = (cq.double() @ t["uq"].to(cuda).T).float()
        parts = torch.stack([q * 0.25, q * 0.75])
        q_plain = torch.empty(n, H * D, device=cuda, dtype=dtype)
        q_full = torch.empty(n, H * (C + R), device=cuda, dtype=dtype)
        ops.latent_prepare(parts, None, *common, q_plain, q_full, None, H, D, R, C)
        ops.head_product(q_plain, D, uk_t, q_full, C + R)
        mixed = torch.empty(n, H * C, device=cuda, dtype=dtype)
        if ops.latent_prompt_usable(q_full, C, R):
            tpt = ops.latent_prompt_tokens(H)
            dev = lambda x: torch.tensor(x, dtype=torch.int32, device=cuda)      # noqa: E731
            if n == 1 and at % 2:                      # every second single token with its pages dealt to two blocks
                per = (min(table.shape[1], ((window or 10 ** 6) + 62) // 64 + 1) + 1) // 2
                partial = torch.full((2, 1, H, C + 2), float("nan"), device=cuda)
                ops.latent_prompt(q_full, kp, mixed, table, dev([0]), dev([0]), 1, a["seq_row0"], a["seq_start"], a["seq_new"], H, C, R,
                                  0.5, None, None, 0, partial, per, window or 0)
            else:
                q0 = list(range(0, n, tpt))
                ops.latent_prompt(q_full, kp, mixed, table, dev([0] * len(q0)), dev(q0), len(q0), a["seq_row0"], a["seq_start"],
                                  a["seq_new"], H, C, R, 0.5, window=window or 0)
        else:
            ops.window_attention(q_full, kp, kp, table, a["row_seq"], a["row_pos"], None, None, None, 0, mixed, H, 1, C + R, C,
                                 window or 0, 0.5, values_in_keys=True)
        out = torch.full((n, H * Dv + 8), 7.0, device=cuda, dtype=dtype)
        ops.head_product(mixed, C, uv, out[:, 8:], Dv)
        got.append(out[:, 8:].cpu())
    got = torch.cat(got).double()
    assert torch.isfinite(got).all()
    assert float((got - ref).abs().max()) < tol * max(1.0, float(ref.abs().max()))


def _delta_rows(gen, T, H, D, Dv):
    return {"r": torch.randn(T, H * D, generator=gen), "k": torch.randn(T, H * D, generator=gen), "v": torch.randn(T, H * Dv, generator=gen),
            "a": torch.randn(T, H * D, generator=gen) * 2, "g": torch.randn(T, H * Dv, generator=gen)}


def _delta_scan(cuda, rows, narrow, t, rate, state, a, H, D, Dv, splits, made_here, chunked=False):
    """The preparing kernel and the scan on the given rows, token by token or by chunks of 16; the projections' sums in
    ``splits`` shares."""
    from camelid_b200.csrc import ops
    n = rows["r"].shape[0]
    proj = torch.cat([rows[x] for x in "rkvag"] + [narrow], 1)
    if splits > 1:
        shares = torch.linspace(0.5, 1.5, splits)
        proj = proj[None] * (shares / shares.sum())[:, None, None]
    packed = torch.empty(n, H, 4 * D + Dv, device=cuda)
    scal = torch.empty(n, H, 4, device=cuda)
    gate = torch.empty(n, H * Dv, device=cuda)
    out = torch.empty(n, H * Dv, device=cuda)
    high = None
    if chunked or not made_here:
        low = torch.empty(n, narrow.shape[1], device=cuda)
        ops.tanh_columns(proj.to(cuda), 3 * H * D + 2 * H * Dv, low)
        high = (low.double() @ t["w2"].double().to(cuda).T).float()
    if chunked:
        dev = lambda x: torch.tensor(x, dtype=torch.int32, device=cuda)      # noqa: E731
        tiles = [(s, q0) for s, k in enumerate(a["seq_new"].tolist()) for q0 in range(0, k, ops.DELTA_CHUNK)]
        chunks = torch.full((len(tiles), H, ops.delta_chunk_floats(D, Dv)), float("nan"), device=cuda)
        ops.delta_chunks(proj.to(cuda), high, t["a.b"].to(cuda), t["w0"].to(cuda), rate, dev([x[0] for x in tiles]), dev([x[1] for x in tiles]),
                         len(tiles), a["seq_row0"], a["seq_new"], chunks, H, D, Dv, gate)
        ops.delta_chunk_scan(chunks, state, a["seq_row0"], a["seq_new"], a["seq_start"], a["seq_slot"], out, len(a["seq_new"]), H, D, Dv)
        return out.cpu(), gate.cpu()
    ops.delta_inputs(proj.to(cuda), t["a.b"].to(cuda), t["w0"].to(cuda), rate, packed, scal, H, D, Dv, high, t["w2"].to(cuda) if made_here else None,
                     gate)
    ops.general_delta_scan(packed, scal, state, a["seq_row0"], a["seq_new"], a["seq_start"], a["seq_slot"], out, len(a["seq_new"]), H, D, Dv)
    return out.cpu(), gate.cpu()


@pytest.mark.parametrize("H,D,Dv,rank", [(3, 24, 24, 8), (1, 128, 128, 6), (2, 20, 7, 16), (2, 33, 33, 5), (1, 200, 64, 40), (4, 3, 5, 8), (2, 64, 64, 24),
                                         (3, 28, 36, 8), (1, 256, 20, 8), (2, 100, 104, 8), (5, 4, 4, 8)])
@pytest.mark.parametrize("chunked", [False, True])
def test_delta_rule_through_portions_and_slots(cuda, H, D, Dv, rank, chunked):
    """Two sequences side by side in portions that differ, in slots that held other states: a key written at row 2 with
    decays near one and removals near zero is asked for at row 140, a head that removes and decays has lost it. Token by
    token, and by chunks of 16 (the portions end inside, at and behind a chunk's edge; single tokens in between)."""
    from camelid_b200.csrc import ops
    if chunked and not ops.delta_chunks_usable(D, Dv):
        return                                                          # odd sizes are walked token by token
    gen = torch.Generator().manual_seed(6)
    T, rate = 150, float(np.exp(-0.5))
    t = {"w2": torch.randn(H * D, rank, generator=gen) * 0.3, "w0": torch.randn(H * D, generator=gen), "a.b": torch.randn(H * D, generator=gen)}
    t["w0"][:D] = -9.0                                                   # head 0 keeps: decay near one, removal near zero
    t["a.b"][:D] = -9.0
    seqs, refs = [], []
    for s in range(2):
        rows, narrow = _delta_rows(gen, T, H, D, Dv), torch.randn(T, rank, generator=gen)
        rows["k"].view(T, H, D)[2, 0] *= 6.0
        rows["r"].view(T, H, D)[140, 0] = rows["k"].view(T, H, D)[2, 0]
        w = np.exp(-rate * pr.sigmoid(np.tanh(narrow.double().numpy()) @ t["w2"].double().numpy().T + t["w0"].double().numpy()))
        a = pr.sigmoid(rows["a"].double().numpy() + t["a.b"].double().numpy())
        n = {x: rows[x].double().numpy() for x in "rkv"}
        ref = pr.delta_core(n["r"], n["k"], n["v"], w, a, H)
        lost = pr.delta_core(n["r"][3:], n["k"][3:], n["v"][3:], w[3:], a[3:], H)        # without the first three writes
        assert np.abs(lost[137, 0] - ref[140, 0]).max() > 1.0
        seqs.append((rows, narrow))
        refs.append(torch.from_numpy(ref.reshape(T, -1)))
    state = torch.full((4, H, Dv, D), 7.0, device=cuda)                 # slots that held something else
    plans = [list(portions(T, c)) for c in ([70, 2, 33, 1, 1], [7, 16, 17, 64, 3])]
    got, at, step = [[], []], [0, 0], 0
    while at[0] < T or at[1] < T:
        live = [s for s in range(2) if at[s] < T]
        news = [next(n for a0, n in plans[s] if a0 == at[s]) for s in live]
        a = arrays(cuda, [at[s] for s in live], news, slots=[3 - s for s in live])
        rows = {x: torch.cat([seqs[s][0][x][at[s]:at[s] + n] for s, n in zip(live, news)]) for x in "rkvag"}
        narrow = torch.cat([seqs[s][1][at[s]:at[s] + n] for s, n in zip(live, news)])
        out, gate = _delta_scan(cuda, rows, narrow, t, rate, state, a, H, D, Dv, 1 + step % 4, step % 2 == 0,
                                chunked and (max(news) > 1 or step % 2 == 0))
        assert torch.allclose(gate, rows["g"], atol=1e-5)
        r0 = 0
        for s, n in zip(live, news):
            got[s].append(out[r0:r0 + n])
            r0 += n
            at[s] += n
        step += 1
    for s in range(2):
        g = torch.cat(got[s]).double()
        assert torch.isfinite(g).all()
        assert float((g - refs[s]).abs().max()) < 5e-5 * float(refs[s].abs().max()), s


def test_delta_rule_with_bfloat16_narrow_weights(cuda):
    """The decays' second matrix in bfloat16, rows read in 16-byte pieces and singly."""
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(8)
    for H, D, rank in ((2, 24, 16), (1, 40, 12)):
        n = 5
        rows, narrow = _delta_rows(gen, n, H, D, D), torch.randn(n, rank, generator=gen)
        w2, w0, ab = torch.randn(H * D, rank, generator=gen).to(torch.bfloat16), torch.randn(H * D, generator=gen), torch.randn(H * D, generator=gen)
        packed, scal = torch.empty(n, H, 5 * D, device=cuda), torch.empty(n, H, 4, device=cuda)
        ops.delta_inputs(torch.cat([rows[x] for x in "rkvag"] + [narrow], 1).to(cuda), ab.to(cuda), w0.to(cuda), 0.4, packed, scal, H, D, D,
                         None, w2.to(cuda))
        w = np.exp(-0.4 * pr.sigmoid(np.tanh(narrow.double().numpy()) @ w2.double().numpy().T + w0.double().numpy())).reshape(n, H, D)
        assert float((packed[:, :, 2 * D:3 * D].cpu().double() - torch.from_numpy(w)).abs().max()) < 1e-5
        a = pr.sigmoid((rows["a"] + ab).double().numpy()).reshape(n, H, D)
        r, k = rows["r"].double().numpy().reshape(n, H, D), rows["k"].double().numpy().reshape(n, H, D)
        n2 = 1.0 / ((k * k).sum(-1) + 1e-6)
        want = np.stack([n2, n2 * (r * a * k).sum(-1), (r * k).sum(-1)], -1)
        assert float((scal[:, :, :3].cpu().double() - torch.from_numpy(want)).abs().max()) < 1e-4


@pytest.mark.parametrize("E,top,splits", [(7, 2, 1), (16, 3, 4), (5, 5, 1), (40, 1, 2), (70, 6, 3)])
def test_routing_with_a_bias_in_the_logits(cuda, E, top, splits):
    """The bias counts for the choice and for the weights; the weights are the softmax over the chosen logits; the logits
    stand in rows that have one more column (the shared expert's gate)."""
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(9)
    rows = 130
    parts = torch.randn(splits, rows, E + 1, generator=gen)
    bias = torch.randn(E, generator=gen) * 3
    ids = torch.empty(rows * top, dtype=torch.int32, device=cuda)
    wts = torch.empty(rows * top, device=cuda)
    ops.route_topk(parts.to(cuda)[..., :E], top, True, True, ids, wts, bias=bias.to(cuda))
    h = parts.sum(0)[:, :E].double().numpy()
    chosen, weights = pr.route(h, {"router": np.eye(E), "router.b": bias.double().numpy()}, E, top)
    assert np.array_equal(ids.cpu().numpy().reshape(rows, top), chosen)
    assert float((wts.cpu().double().view(rows, top) - torch.from_numpy(weights)).abs().max()) < 1e-5


@pytest.mark.parametrize("hidden,splits", [(64, 1), (37, 3), (1024, 2)])
def test_combining_with_a_gated_shared_expert_into_the_stream(cuda, hidden, splits):
    from camelid_b200.csrc import ops
    gen = torch.Generator().manual_seed(10)
    rows, top, E = 9, 2, 3
    y = torch.randn(rows * top, hidden, generator=gen)
    place = torch.randperm(rows * top, generator=gen).to(torch.int32)
    wts = torch.rand(rows * top, generator=gen)
    shared, logits = torch.randn(splits, rows, hidden, generator=gen), torch.randn(splits, rows, E + 1, generator=gen)
    stream = torch.randn(rows, hidden, generator=gen)
    sg = torch.sigmoid(logits.sum(0)[:, E].double())
    ref = shared.sum(0).double() * sg[:, None] + (y[place.long()].double() * wts[:, None].double()).view(rows, top, hidden).sum(1)
    for accumulate in (False, True):
        out = stream.to(cuda).clone()
        ops.expert_combine(y.to(cuda), place.to(cuda), wts.to(cuda), top, True, shared.to(cuda), out, None, logits.to(cuda)[..., E:], accumulate)
        want = ref + stream.double() if accumulate else ref
        assert float((out.cpu().double() - want).abs().max()) < 1e-5
