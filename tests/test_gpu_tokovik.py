"""Tokovik on the GPU against the plain evaluation (tests/plain_tokovik.py): every mechanism, prompts, portions, decoding, window
edges, rings that wrap, batches, slots that are used again, generation through the scheduler and the command lines."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import layered_helpers as lh
import tokovik_cases as tc
from helpers import has_gpu
from layered_helpers import DTYPES, LIMIT, check, cut, feed, rel_rms, tokens

pytestmark = [pytest.mark.gpu, pytest.mark.skipif(not has_gpu(), reason="needs a GPU")]
ROOT = Path(__file__).resolve().parent.parent


# ---------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", sorted(tc.CASES))
def test_prompt_portions_and_decoding_follow_the_plain_evaluation(case, dtype):
    cfg = tc.CASES[case]
    params = tc.random_params(cfg, 7)
    n = 150
    toks = tokens(cfg, n, 8)
    ref, ref_taps = tc.plain(params, cfg, toks)
    eng = tc.engine(cfg, params, max_pos=n + 3, max_seqs=2, dtype=dtype)
    runs = eng.layer_runs()
    logits, taps = feed(eng, 0, toks, [n], taps=runs)
    for r in range(runs):
        check(taps[r], ref_taps[r], dtype, f"residual after layer {r}")
    check(logits, ref, dtype, "whole")
    for parts in ([1] * n, cut(n, [2]), cut(n, [3, 17, 2, 65]), cut(n, [64]), [100, 2] + [1] * 48, [31, 33, 86], [1, 149], cut(n, [15, 16])):
        check(feed(eng, 1, toks, parts), ref, dtype, parts[:4])
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("part", ["left", "right", "mlp"])
def test_each_part_alone(part, dtype):
    """A branch whose output norm is zero gives nothing; a feed-forward norm stored as -1 gives nothing."""
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 9)
    for name in params:
        off = (".left.out" in name and part != "left") or (".right.out" in name and part != "right")
        if off:
            params[name] = np.zeros_like(params[name])
        if name.endswith("norm2") and part != "mlp":
            params[name] = -np.ones_like(params[name])
        if name.endswith("norm1") and part == "mlp":
            params[name] = -np.ones_like(params[name])
    toks = tokens(cfg, 100, 10)
    ref, ref_taps = tc.plain(params, cfg, toks)
    eng = tc.engine(cfg, params, max_pos=100, dtype=dtype)
    for parts in ([100], [97] + [1] * 3, cut(100, [2]), cut(100, [40])):
        logits, taps = feed(eng, 0, toks, parts, taps=eng.layer_runs())
        check(logits, ref, dtype, parts[:3])
        for r in range(len(taps)):
            check(taps[r], ref_taps[r], dtype, (r, parts[:3]))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [5, 24, 70])
def test_rings_that_wrap(portion, dtype):
    """Steps of few rows leave the caches little more than the window: positions share rows many times over."""
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 13)
    n = 260
    toks = tokens(cfg, n, 14)
    ref, _ = tc.plain(params, cfg, toks)
    eng = tc.engine(cfg, params, max_pos=n, max_seqs=2, dtype=dtype, portion=portion)
    for slot, parts in ((1, [n]), (0, cut(n, [portion])), (1, cut(n, [2, portion, 1, 7])), (0, [n - 60] + [1] * 60)):
        check(feed(eng, slot, toks, parts), ref, dtype, (portion, parts[:4]))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 17)
    toks = tokens(cfg, 700, 18)
    ref, _ = tc.plain(params, cfg, toks)
    eng = tc.engine(cfg, params, max_pos=720, dtype=dtype, portion=8)
    eng.extend(0, toks[:3], 0)
    got = []
    for i in range(3, 700):
        _, logits, _ = eng.step_batch([0], [toks[i]], [i], want_logits=True)
        got.append(logits[0])
    check(np.array(got), ref[3:], dtype, "decoded")
    assert eng.filled(0) == 700
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_longer_than_a_step(dtype):
    """More tokens than one step's rows, and more wanted places than the logits buffer holds."""
    cfg = tc.config([tc.layer(tc.left(heads=4, window=600, dims=12), tc.right(heads=2, dim=16), 40)], width=48, vocab=64)
    params = tc.random_params(cfg, 27)
    n = 2100
    toks = tokens(cfg, n, 28)
    ref, _ = tc.plain(params, cfg, toks)
    eng = tc.engine(cfg, params, max_pos=n, dtype=dtype)
    want = list(range(0, n, 13)) + [n - 1]
    check(eng.extend(0, toks, 0, want)[1], ref[want], dtype, "sparse places")
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decays_from_none_to_all(dtype):
    """Channels that forget everything at once beside channels that forget nothing, and others that turn from one to the
    other from token to token: no exponential overflows, nothing that must stay is lost."""
    cfg = tc.config([tc.layer(tc.left(window=5), tc.right(heads=2, dim=40, vdim=24, tau=1.0), 0)] * 2, width=80, rank=4)
    params = tc.random_params(cfg, 31)
    rng = np.random.default_rng(32)
    for i in range(2):
        params[f"l{i}.mix.right.a2.b"] = rng.choice([-90.0, -30.0, 0.0, 8.0, 30.0], 80)
        params[f"l{i}.mix.right.a2"] *= 12.0
        params[f"l{i}.mix.left.out"] *= 0.2
    params = tc.rounded(params)
    toks = tokens(cfg, 200, 33)
    ref, _ = tc.plain(params, cfg, toks)
    eng = tc.engine(cfg, params, max_pos=200, dtype=dtype)
    for parts in ([200], cut(200, [64]), cut(200, [50, 1, 2]), [130] + [1] * 70):
        check(feed(eng, 0, toks, parts), ref, dtype, parts[:3], 1.5)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence(dtype):
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 47)
    eng = tc.engine(cfg, params, max_pos=40, dtype=dtype)
    for n in (1, 2, 3, 4, 5, 17):
        toks = tokens(cfg, n, 50 + n)
        ref, _ = tc.plain(params, cfg, toks)
        check(feed(eng, 0, toks, [n]), ref, dtype, n)
        check(feed(eng, 0, toks, [1] * n), ref, dtype, n)
    eng.close()


# ---------------------------------------------------------------- one key among many

A, B = 5, 9  # the token that is looked for, and the one that looks


def window_needle(window, per=2):
    """A window in which token A's key answers token B's query far above all others."""
    cfg = tc.config([tc.layer(tc.left(heads=2 * per, kv_heads=2, dim=64, vdim=24, window=window, dims=2, base=100.0, scaling=None, scale=28.0 / 64),
                              tc.right(), 0)], width=104, vocab=90, embed=0.5)
    p = tc.random_params(cfg, 37)
    h = p["embed"] * cfg["embedding"]["scale"]
    u = np.where(np.arange(64) < 2, 0.0, np.random.default_rng(1).choice([-1.0, 1.0], 64))
    only = lambda t: np.linalg.lstsq(h, np.where(np.arange(90) == t, 1.0, 0.0), rcond=None)[0]  # noqa: E731
    for name, heads, tok in (("q", 2 * per, B), ("k", 2, A)):
        p[f"l0.mix.left.{name}"] += 6.0 * np.outer(np.tile(u, heads), only(tok))
        p[f"l0.mix.left.{name}.b"] *= 0.3
        p[f"l0.mix.left.{name}.norm"] = np.ones(64)
    p["l0.mix.right.out"] *= 0.1
    return cfg, tc.rounded(p)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,per", [(2, 2), (16, 1), (17, 2), (40, 20), (64, 4), (65, 2), (130, 3), (170, 2)])
def test_window_edges(window, per, dtype):
    """The key at the window's last place counts and the one before it does not, in prompts, portions and decoding, wherever the
    query lies; rings of the smallest size included."""
    cfg, params = window_needle(window, per)
    wider, narrower = copy.deepcopy(cfg), copy.deepcopy(cfg)
    wider["layers"][0]["mixer"]["left"]["mask"]["size"] = window + 1
    narrower["layers"][0]["mixer"]["left"]["mask"]["size"] = window - 1
    rng = np.random.default_rng(38)
    limit = 1.5 * LIMIT[dtype]
    engines = [tc.engine(cfg, params, max_pos=440, dtype=dtype), tc.engine(cfg, params, max_pos=440, dtype=dtype, portion=19)]
    for n in (window + 1, window + 2, window + 63, 2 * window + 70):
        for back, other in ((window - 1, narrower), (window, wider), (1, None)):
            toks = rng.integers(10, 90, n).tolist()
            toks[-1], toks[n - 1 - back] = B, A
            ref, _ = tc.plain(params, cfg, toks)
            if other:
                wrong, _ = tc.plain(params, other, toks)
                assert rel_rms(wrong[-1:], ref[-1:])[0] > 4 * limit, "the case does not show the edge"
            for parts in ([n], [n - 1, 1], [n - 2, 2], cut(n, [64]), [n - back, back], [n - min(20, n - 1)] + [1] * min(20, n - 1)):
                for eng in engines:
                    got = feed(eng, 0, toks, [k for k in parts if k])
                    assert rel_rms(got[-1:], ref[-1:])[0] <= limit, (n, back, parts[:3])
    for eng in engines:
        eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_stays_in_the_state(dtype):
    """A head that forgets nothing takes in token A and, next to it, no other; token B reads it."""
    cfg = tc.config([tc.layer(tc.left(window=3), tc.right(heads=2, dim=16, vdim=24, tau=16.0), 0)], width=96, vocab=80, rank=6, embed=0.5)
    p = tc.random_params(cfg, 41)
    h = p["embed"] * cfg["embedding"]["scale"]
    only = lambda t: np.linalg.lstsq(h, np.where(np.arange(80) == t, 1.0, 0.0), rcond=None)[0]  # noqa: E731
    u = np.ones(16)
    p["l0.mix.right.q"][:16], p["l0.mix.right.k"][:16] = np.outer(u, 3.0 * only(B)), np.outer(u, 3.0 * only(A))
    p["l0.mix.right.a2"][:16], p["l0.mix.right.a2.b"][:16] = 0.0, 14.0
    p["l0.mix.left.out"] *= 0.1
    p = tc.rounded(p)
    rng = np.random.default_rng(42)
    limit = 1.5 * LIMIT[dtype]
    eng = tc.engine(cfg, p, max_pos=320, dtype=dtype)
    for n, places in ((70, (0, 1, 15, 16, 17, 47, 48, 62, 63, 64, 65, 68)), (300, (0, 2, 127, 128, 191, 192, 255, 256, 257, 298))):
        fill = rng.integers(10, 80, n).tolist()
        fill[-1] = B
        without, _ = tc.plain(p, cfg, fill)
        for at in places:
            toks = list(fill)
            toks[at] = A
            ref, _ = tc.plain(p, cfg, toks)
            assert rel_rms(without[-1:], ref[-1:])[0] > 4 * limit, "the case does not show the token"
            for parts in ([n], [n - 1, 1], cut(n, [64]), [at + 1] + cut(n - at - 1, [2]), [n - 40] + [1] * 40):
                got = feed(eng, 0, toks, parts)
                assert rel_rms(got[-1:], ref[-1:])[0] <= limit, (n, at, parts[:3])
    eng.close()


# ---------------------------------------------------------------- slots and batches

@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests_equal_each_alone(dtype):
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 57)
    slots = 20
    eng = tc.engine(cfg, params, max_pos=140, max_seqs=slots, dtype=dtype, portion=24)
    lengths = [(7 * i) % 90 + 1 for i in range(slots)]
    seqs = {s: tokens(cfg, n + 8, 60 + s) for s, n in enumerate(lengths)}
    refs = {s: tc.plain(params, cfg, t)[0] for s, t in seqs.items()}
    for s, n in enumerate(lengths):
        eng.extend(s, seqs[s][:n], 0)
    at = dict(enumerate(lengths))
    rng = np.random.default_rng(61)
    for size in (20, 1, 2, 3, 5, 20, 9, 17):
        rows = [s for s in rng.permutation(slots) if at[s] < len(seqs[s])][:size]
        _, logits, _ = eng.step_batch(rows, [seqs[s][at[s]] for s in rows], [at[s] for s in rows], want_logits=True)
        check(logits, np.array([refs[s][at[s]] for s in rows]), dtype, rows)
        for s in rows:
            at[s] += 1
    # several greedy steps at once, fed back on the device, against one at a time
    rows, cur = [3, 0, 7], [1, 2, 3]
    got = eng.decode_greedy(rows, cur, [at[s] for s in rows], 6)
    for i, s in enumerate(rows):
        lh.greedy_follows(tc.plain, params, cfg, seqs[s][:at[s]] + [cur[i]], got[:, i], dtype)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_are_used_again_and_sequences_cannot_be_rewound(cm, dtype):
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 67)
    eng = tc.engine(cfg, params, max_pos=100, max_seqs=2, dtype=dtype, portion=16)
    a, b = tokens(cfg, 90, 68), tokens(cfg, 40, 69)
    ref_a, ref_b = tc.plain(params, cfg, a)[0], tc.plain(params, cfg, b)[0]
    feed(eng, 0, a, [90])
    feed(eng, 1, a, [70, 20])
    check(feed(eng, 0, b, [1, 39]), ref_b, dtype, "a slot that held a longer sequence")
    check(feed(eng, 1, b, cut(40, [1, 2, 33])), ref_b, dtype, "the other slot")
    check(feed(eng, 0, a, [64, 26]), ref_a, dtype, "and the first again")
    for call in (lambda: eng.extend(0, [1], 89), lambda: eng.extend(0, [1, 2], 91), lambda: eng.step_batch([1], [1], [39]),
                 lambda: eng.extend(0, [1] * 11, 90)):
        with pytest.raises(cm.CmldError):
            call()
    assert eng.filled(0) == 90 and eng.filled(1) == 40
    check(feed(eng, 1, a, [90]), ref_a, dtype, "after refused calls")
    eng.close()


def test_tensors_are_those_of_the_design(cm):
    cfg = tc.CASES["unequal_layers"]
    eng = tc.engine(cfg, tc.random_params(cfg, 1), max_pos=8)
    assert eng.tensors() == tc.tensor_shapes(cfg) and eng.weights_ready()
    eng.close()


# ---------------------------------------------------------------- generation through the framework's own entry points

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [0, 2, 40])
def test_greedy_generation_through_the_scheduler(dtype, portion, tmp_path):
    from camelid_b200 import models
    from camelid_b200.scheduler import Scheduler

    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 77)
    eng = models.load_model(lh.write_folder(tmp_path / "m", cfg, params), max_pos=128, max_seqs=3, dtype=dtype)
    s = Scheduler(eng, portion=portion, greedy_run=4)
    prompts = {i: tokens(cfg, n, 80 + i) for i, n in enumerate((50, 1, 70, 3, 33))}
    for i, p in prompts.items():
        s.submit(i, p, 6 + 2 * i)
    s.submit("drawn", [1, 2, 3], 5, temperature=2.0, seed=3)
    out = s.run()
    for i, p in prompts.items():
        assert len(out[i]) == 6 + 2 * i
        lh.greedy_follows(tc.plain, params, cfg, p, out[i], dtype)
    assert len(out["drawn"]) == 5
    eng.close()


def test_command_lines(tmp_path):
    cfg = tc.CASES["unequal_layers"]
    params = tc.random_params(cfg, 97)
    folder = lh.write_folder(tmp_path / "m", cfg, params)
    toks = tokens(cfg, 30, 98)
    ref, _ = tc.plain(params, cfg, toks)
    r = subprocess.run([sys.executable, "-m", "camelid_b200.generate", "--model", str(folder), "--dtype", "float32", "-n", "5", "--tokens",
                        ",".join(map(str, toks)), "--tokens", "1,2"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    lines = r.stdout.strip().splitlines()
    assert len(lines) == 2
    lh.greedy_follows(tc.plain, params, cfg, toks, [int(t) for t in lines[0].split(",")], "float32")
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:11], "want": [0, 10]}], "end": []},
                 {"step": 1, "entries": [{"id": "x", "tokens": toks[11:13], "want": []}], "end": []},
                 {"step": 2, "entries": [{"id": "x", "tokens": toks[13:], "want": [1, 16]}], "end": ["x"]},
                 {"step": 3, "entries": [{"id": "z", "tokens": toks[:1], "want": [0]}], "end": ["z"]}]
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "3.f32"]
        for step, places in ((0, [0, 10]), (2, [14, 29]), (3, [0])):
            check(np.fromfile(out / f"{step}.f32", "<f4").reshape(-1, cfg["vocab"]), ref[places], dtype, step)
