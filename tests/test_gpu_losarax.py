"""Losarax on the GPU against the plain evaluation (tests/plain_losarax.py): every mechanism, prompts, portions, decoding,
batches, slots that are used again, generation through the scheduler and the command lines."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest

import losarax_cases as lc
import plain_losarax as pl
import layered_helpers as lh
from helpers import has_gpu
from layered_helpers import DTYPES, check, cut, feed

pytestmark = [pytest.mark.gpu, pytest.mark.skipif(not has_gpu(), reason="needs a GPU")]
ROOT = Path(__file__).resolve().parent.parent


# ---------------------------------------------------------------- the linear layers alone

LIN_SHAPES = [  # out, in, rows: edges of tiles, of clusters that share a tile, of padding
    (128, 64, 16), (1, 8, 3), (130, 72, 5), (300, 515, 33), (257, 1000, 64), (96, 4096, 20), (1024, 256, 65), (515, 130, 129), (2000, 320, 300),
    (4096, 192, 700), (640, 2048, 257)]


def device_rows(a, bf16):
    """Rows padded to a multiple of eight columns, on the device."""
    from camelid_b200.engine import DeviceBuffer
    from camelid_b200.safetensors import to_bf16

    ld = (a.shape[1] + 7) // 8 * 8
    p = np.zeros((a.shape[0], ld), np.float32)
    p[:, :a.shape[1]] = a
    return DeviceBuffer.from_numpy(to_bf16(p) if bf16 else p)


def linear(cm, kernel, w, x, out_bf16=False, act=0, act_rows=0, bias=None, scale=1.0):
    import ctypes as C

    from camelid_b200._lib import check as ok
    from camelid_b200.engine import DeviceBuffer
    from camelid_b200.safetensors import from_bf16

    wd, xd = device_rows(w, True), device_rows(x, kernel == 1)
    outs = w.shape[0] // 2 if act == 3 else w.shape[0]
    out = DeviceBuffer(x.shape[0] * outs * (2 if out_bf16 else 4))
    bd = None if bias is None else DeviceBuffer.from_numpy(np.asarray(bias, np.float32))
    ms = C.c_float(0)
    ok(cm.lib().cmld_linear(kernel, wd.ptr, w.shape[0], w.shape[1], xd.ptr, x.shape[0], out.ptr, int(out_bf16), act, act_rows,
                            bd.ptr if bd else None, scale, 1, 0, C.byref(ms)))
    y = out.to_numpy(np.uint16 if out_bf16 else np.float32)
    return (from_bf16(y) if out_bf16 else y).reshape(x.shape[0], outs)


def lin_case(shape, seed=0):
    from camelid_b200.safetensors import from_bf16, to_bf16

    rng = np.random.default_rng(seed)
    o, k, n = shape
    w, x = rng.standard_normal((o, k)) / np.sqrt(k), rng.standard_normal((n, k))
    return from_bf16(to_bf16(w)).reshape(o, k), from_bf16(to_bf16(x)).reshape(n, k)


@pytest.mark.parametrize("shape", LIN_SHAPES)
def test_linear_kernels(cm, shape):
    w, x = lin_case(shape)
    ref = x.astype(np.float64) @ w.astype(np.float64).T
    for kernel in (1, 2):
        assert np.abs(linear(cm, kernel, w, x) - ref).max() < 2e-5, kernel
    assert np.abs(linear(cm, 1, w, x, out_bf16=True) - ref).max() < 2e-2 * max(1.0, np.abs(ref).max())
    for n in (1, 2):
        assert np.abs(linear(cm, 0, w, x[:n]) - ref[:n]).max() < 2e-5


def test_linear_activations(cm):
    w, x = lin_case((200, 96, 40), 3)
    ref = x.astype(np.float64) @ w.astype(np.float64).T
    silu = ref.copy()
    silu[:, :70] = pl.silu(ref[:, :70])
    for kernel, rows in ((0, 2), (1, 40), (2, 40)):
        assert np.abs(linear(cm, kernel, w, x[:rows], act=1, act_rows=70) - silu[:rows]).max() < 5e-5
        assert np.abs(linear(cm, kernel, w, x[:rows], act=2) - np.maximum(ref[:rows], 0) ** 2).max() < 1e-4


@pytest.mark.parametrize("shape", [(200, 96, 40), (130, 1024, 5), (2, 8, 3), (258, 72, 64), (514, 320, 129), (1026, 256, 300)])
def test_linear_gated_pairs_bias_and_scale(cm, shape):
    """Tiles, clusters that share a tile, odd row counts; bias and factor before the activation."""
    w, x = lin_case(shape, 5)
    b = np.random.default_rng(6).standard_normal(shape[0]).astype(np.float32)
    ref = 0.7 * (x.astype(np.float64) @ w.astype(np.float64).T) + b
    pair = pl.silu(ref[:, 0::2]) * ref[:, 1::2]
    for kernel, rows in ((0, 1), (0, 2), (1, shape[2]), (2, shape[2])):
        assert np.abs(linear(cm, kernel, w, x[:rows], bias=b, scale=0.7) - ref[:rows]).max() < 5e-5, kernel
        assert np.abs(linear(cm, kernel, w, x[:rows], act=3, bias=b, scale=0.7) - pair[:rows]).max() < 2e-4, kernel
    assert np.abs(linear(cm, 1, w, x, out_bf16=True, act=3, bias=b, scale=0.7) - pair).max() < 2e-2 * max(1.0, np.abs(pair).max())


# ---------------------------------------------------------------- whole models

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", sorted(lc.CASES))
def test_prompt_portions_and_decoding_follow_the_plain_evaluation(case, dtype):
    cfg = lc.CASES[case]
    params = lc.random_params(cfg, 7)
    n = 150
    toks = lc.tokens(cfg, n, 8)
    ref, ref_taps = lc.plain(params, cfg, toks)
    eng = lc.engine(cfg, params, max_pos=n + 3, max_seqs=2, dtype=dtype)
    runs = eng.layer_runs()
    logits, taps = feed(eng, 0, toks, [n], taps=runs)
    for r in range(runs):
        check(taps[r], ref_taps[r], dtype, f"residual after run {r}", 1.0 if dtype == "float32" else 1.5)
    check(logits, ref, dtype, "whole")
    for parts in ([1] * n, cut(n, [2]), cut(n, [3, 17, 2, 65]), cut(n, [64]), [100, 2] + [1] * 48, [31, 33, 86], [1, 149]):
        check(feed(eng, 1, toks, parts), ref, dtype, parts[:4])
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """A few prompt tokens, then hundreds of single tokens, past the places where a step takes another launch shape."""
    cfg = lc.CASES["both_mlp_on_lightning"]
    params = lc.random_params(cfg, 17)
    toks = lc.tokens(cfg, 600, 18)
    ref, _ = lc.plain(params, cfg, toks)
    eng = lc.engine(cfg, params, max_pos=640, dtype=dtype)
    eng.extend(0, toks[:3], 0)
    got = []
    for i in range(3, 600):
        _, logits, _ = eng.step_batch([0], [toks[i]], [i], want_logits=True)
        got.append(logits[0])
    check(np.array(got), ref[3:], dtype, "decoded")
    assert eng.filled(0) == 600
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_portions_longer_than_a_step(dtype):
    """More tokens than one step's rows, and more wanted places than the logits buffer holds."""
    cfg = lc.config([lc.with_mlp(lc.latent(heads=2, dim=16, vdim=8, q_rank=24, kv_rank=32), 40), lc.lightning(heads=2, dim=16, vdim=8, decay=[0.9, 1.0])],
                    width=48, vocab=64)
    params = lc.random_params(cfg, 27)
    n = 2100
    toks = lc.tokens(cfg, n, 28)
    ref, _ = lc.plain(params, cfg, toks)
    eng = lc.engine(cfg, params, max_pos=n, dtype=dtype)
    want = list(range(0, n, 13)) + [n - 1]
    _, logits = eng.extend(0, toks, 0, want)
    check(logits, ref[want], dtype, "sparse places")
    eng.close()


# ---------------------------------------------------------------- one key among many

def latent_needle(seed):
    """A latent layer in which token A's key answers token B's query far above all others, whatever lies between."""
    cfg = lc.config([lc.latent(heads=2, dim=16, vdim=24, q_rank=64, kv_rank=80, rot_dim=8)], width=96, vocab=120, streams=2)
    p = lc.random_params(cfg, seed)
    a, b = 5, 9
    s_in = p["l0.hc1.in"].sum()
    h = pl.layer_norm(s_in * pl.layer_norm(p["embed"], p["embed.norm"], p["embed.norm.b"], 1e-5), p["l0.norm1"], p["l0.norm1.b"], 1e-5)
    cq = pl.rms_norm(pl.linear(p["l0.mix.dq"], h[b]), p["l0.mix.dq.norm"], 1e-5)
    c = pl.rms_norm(pl.linear(p["l0.mix.dkv"], h[a])[:80], p["l0.mix.dkv.norm"], 1e-5)
    u = np.ones(16) / 4.0
    g = np.sqrt(40.0 / cfg["layers"][0]["mixer"]["scale"])
    p["l0.mix.uq"][:16] += g * np.outer(u, cq) / (cq @ cq)
    p["l0.mix.uk"][:16] += g * np.outer(u, c) / (c @ c)
    return cfg, p, a, b


def lightning_needle(seed):
    """A lightning layer whose first head never forgets and takes in token A's value and, next to it, no other."""
    cfg = lc.config([lc.lightning(heads=2, dim=16, vdim=24, decay=[1.0, 0.9])], width=96, vocab=80, streams=2)
    p = lc.random_params(cfg, seed)
    a, b = 5, 9
    s_in = p["l0.hc1.in"].sum()
    h = pl.layer_norm(s_in * pl.layer_norm(p["embed"], p["embed.norm"], p["embed.norm.b"], 1e-5), p["l0.norm1"], p["l0.norm1.b"], 1e-5)
    only = lambda t, rest: np.linalg.lstsq(h, np.where(np.arange(80) == t, 1.0, rest), rcond=None)[0]  # noqa: E731
    u = np.ones(16)
    p["l0.mix.q"][:16] = np.outer(u, 3.0 * only(b, -1.0))
    p["l0.mix.k"][:16] = np.outer(u, 3.0 * only(a, -2.0))
    p["l0.mix.v"][:24] += 4.0 * np.outer(np.resize([2.0, 0.5, 1.5], 24), only(a, 0.0))
    return cfg, p, a, b


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("make", [latent_needle, lightning_needle])
def test_a_single_far_key_is_found_wherever_it_lies(make, dtype):
    cfg, params, a, b = make(37)
    from camelid_b200.safetensors import from_bf16, to_bf16

    params = {k: from_bf16(to_bf16(v)).reshape(v.shape) for k, v in params.items()}
    rng = np.random.default_rng(38)
    eng = lc.engine(cfg, params, max_pos=320, dtype=dtype)
    limit = 2 * lc.LIMIT[dtype]
    for n, places in ((70, (0, 1, 31, 32, 33, 62, 63, 64, 65, 68)), (300, (0, 2, 127, 128, 191, 192, 255, 256, 257, 298))):
        fill = rng.integers(10, cfg["vocab"], n).tolist()
        fill[-1] = b
        without, _ = lc.plain(params, cfg, fill)
        for at in places:
            toks = list(fill)
            toks[at] = a
            ref, _ = lc.plain(params, cfg, toks)
            assert lc.rel_rms(without[-1:], ref[-1:])[0] > 4 * limit, "the case does not show the key"
            for parts in ([n], [n - 1, 1], cut(n, [64]), [at + 1] + cut(n - at - 1, [2]), [n - 40] + [1] * 40):
                got = feed(eng, 0, toks, [p for p in parts if p])
                assert lc.rel_rms(got[-1:], ref[-1:])[0] <= limit, (n, at, parts[:3])
        # a key that comes after the query is not seen
        toks = fill[:-1] + [fill[0], a]
        toks[n - 2] = b
        ref, _ = lc.plain(params, cfg, toks)
        got = feed(eng, 0, toks, [len(toks)])
        check(got[n - 2:n - 1], ref[n - 2:n - 1], dtype, "the key after the query", 2.0)
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_of_a_sequence(dtype):
    cfg = lc.CASES["both_mlp_on_lightning"]
    params = lc.random_params(cfg, 47)
    eng = lc.engine(cfg, params, max_pos=40, dtype=dtype)
    for n in (1, 2, 3, 4, 5):
        toks = lc.tokens(cfg, n, 50 + n)
        ref, _ = lc.plain(params, cfg, toks)
        check(feed(eng, 0, toks, [n]), ref, dtype, n)
        check(feed(eng, 0, toks, [1] * n), ref, dtype, n)
    eng.close()


# ---------------------------------------------------------------- slots and batches

@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests_equal_each_alone(dtype):
    """Decode steps of 1, 2, 3, 5, 20 rows (matrix-vector, split and whole tensor-core products), slots in any order."""
    cfg = lc.CASES["both_mlp_on_lightning"]
    params = lc.random_params(cfg, 57)
    slots = 20
    eng = lc.engine(cfg, params, max_pos=140, max_seqs=slots, dtype=dtype)
    lengths = [(7 * i) % 90 + 1 for i in range(slots)]
    seqs = {s: lc.tokens(cfg, n + 8, 60 + s) for s, n in enumerate(lengths)}
    refs = {s: lc.plain(params, cfg, t)[0] for s, t in seqs.items()}
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
    rows = [3, 0, 7]
    cur = [1, 2, 3]
    got = eng.decode_greedy(rows, cur, [at[s] for s in rows], 6)
    for i, s in enumerate(rows):
        toks = seqs[s][:at[s]] + [cur[i]]
        for t in got[:, i]:
            ref = lc.plain(params, cfg, toks)[0][-1]
            assert ref[int(t)] >= ref.max() - 4 * lc.LIMIT[dtype] * np.sqrt((ref ** 2).mean()), (i, int(t))
            toks.append(int(t))
    eng.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_slots_are_used_again_and_sequences_cannot_be_rewound(cm, dtype):
    cfg = lc.CASES["both_mlp_on_lightning"]
    params = lc.random_params(cfg, 67)
    eng = lc.engine(cfg, params, max_pos=100, max_seqs=2, dtype=dtype)
    a, b = lc.tokens(cfg, 90, 68), lc.tokens(cfg, 40, 69)
    ref_a, ref_b = lc.plain(params, cfg, a)[0], lc.plain(params, cfg, b)[0]
    feed(eng, 0, a, [90])
    feed(eng, 1, a, [70, 20])
    check(feed(eng, 0, b, [1, 39]), ref_b, dtype, "a slot that held a longer sequence")
    check(feed(eng, 1, b, cut(40, [1, 2, 33])), ref_b, dtype, "the other slot")
    check(feed(eng, 0, a, [64, 26]), ref_a, dtype, "and the first again")
    for call in (lambda: eng.extend(0, [1], 89), lambda: eng.extend(0, [1, 2], 91), lambda: eng.step_batch([1], [1], [39]),
                 lambda: eng.step_batch([1, 1], [1, 2], [40, 41]), lambda: eng.extend(0, [1] * 11, 90), lambda: eng.extend(0, [cfg["vocab"]], 90),
                 lambda: eng.extend(2, [1], 0), lambda: eng.extend(0, [1, 2], 90, [1, 0])):
        with pytest.raises(cm.CmldError):
            call()
    assert eng.filled(0) == 90 and eng.filled(1) == 40
    check(feed(eng, 1, a, [90]), ref_a, dtype, "after refused calls")
    eng.close()


def test_calls_of_llama_shaped_engines_are_refused(cm):
    cfg = lc.CASES["latent"]
    eng = lc.engine(cfg, lc.random_params(cfg, 1), max_pos=8)
    x = np.zeros(cfg["width"], np.float32)
    out = np.zeros(cfg["vocab"], np.float32)
    rc = cm.lib().cmld_engine_forward_token_logits(eng._h, x.ctypes.data, x.ctypes.data, x.ctypes.data, 0, 1.0, out.ctypes.data)
    assert rc == 3 and b"layered design" in cm.lib().cmld_last_error()
    assert cm.lib().cmld_engine_read_kv_layer(eng._h, 0, 1, x.ctypes.data, x.ctypes.data) == 3
    eng.close()


def test_missing_tensor_is_named(cm):
    from camelid_b200 import losarax
    from camelid_b200.layered import LayeredEngine

    cfg = lc.CASES["latent"]
    eng = LayeredEngine(losarax.spec_from_config(cfg), 8)
    assert not eng.weights_ready()
    assert {k: (v if len(v) == 2 else (int(np.prod(v)),)) for k, v in lc.tensor_shapes(cfg).items() if "mix" not in k.rsplit(".", 1)[-1]} == {
        k: v for k, v in eng.tensors().items() if "mix" not in k.rsplit(".", 1)[-1]}
    with pytest.raises(cm.CmldError, match="embed is not set"):
        eng.extend(0, [1], 0)
    with pytest.raises(cm.CmldError, match="no tensor"):
        eng.set_tensor("l0.mix.nothing", np.zeros(4, np.uint16))
    eng.close()


# ---------------------------------------------------------------- extend and sampling on the llama-shaped engine

def test_extend_and_sample_on_a_llama_shaped_engine(cm, orc):
    from camelid_b200 import synth

    cfg = synth.engine_config("tiny", max_pos=96, max_seqs=2)
    eng = synth.build_engine(cfg, "q4_k_m", 5)
    prompt = orc.synth_tokens(5, 5, 45, cfg.vocab)
    nxt, logits = eng.extend(0, prompt, 0, [0, 7, 33, 44])
    assert nxt == int(np.argmax(logits[-1])) == eng.prefill_tokens(1, prompt, 0)
    one = [eng.extend(1, prompt[i:i + 1], i, [0])[1][0] for i in range(45)]
    assert np.array_equal(logits, np.array(one)[[0, 7, 33, 44]])
    assert eng.sample(1e-4, 3) == nxt
    draws = {eng.sample(5.0, seed) for seed in range(30)}
    assert len(draws) > 5 and eng.sample(5.0, 7) == eng.sample(5.0, 7)
    eng.close()


# ---------------------------------------------------------------- generation through the framework's own entry points

def greedy_follows(params, cfg, prompt, out, dtype):
    lh.greedy_follows(lc.plain, params, cfg, prompt, out, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [0, 2, 40])
def test_greedy_generation_through_the_scheduler(dtype, portion, tmp_path):
    from camelid_b200 import models
    from camelid_b200.scheduler import Scheduler

    cfg = lc.CASES["both_mlp_on_lightning"]
    params = lc.random_params(cfg, 77)
    folder = lc.write_folder(tmp_path / "m", cfg, params)
    eng = models.load_model(folder, max_pos=128, max_seqs=3, dtype=dtype)
    s = Scheduler(eng, portion=portion, greedy_run=4)
    prompts = {i: lc.tokens(cfg, n, 80 + i) for i, n in enumerate((50, 1, 70, 3, 33))}
    for i, p in prompts.items():
        s.submit(i, p, 6 + 2 * i)
    out = s.run()
    for i, p in prompts.items():
        assert len(out[i]) == 6 + 2 * i
        greedy_follows(params, cfg, p, out[i], dtype)
    eng.close()


def test_sampling_through_the_scheduler(tmp_path):
    from camelid_b200 import models
    from camelid_b200.scheduler import Scheduler

    cfg = lc.CASES["both_mlp_on_lightning"]
    folder = lc.write_folder(tmp_path / "m", cfg, lc.random_params(cfg, 87))
    outs = []
    for seed in (1, 1, 2):
        eng = models.load_model(folder, max_pos=64, max_seqs=2)
        s = Scheduler(eng)
        s.submit("hot", [1, 2, 3], 12, temperature=2.0, seed=seed)
        s.submit("cold", [4, 5], 12, temperature=1e-4, seed=seed)
        s.submit("greedy", [4, 5], 12)
        outs.append(dict(s.run()))
        eng.close()
    assert outs[0] == outs[1] and outs[0]["hot"] != outs[2]["hot"]
    assert outs[0]["cold"] == outs[0]["greedy"]


def test_command_lines(tmp_path):
    cfg = lc.CASES["both_mlp_on_lightning"]
    params = lc.random_params(cfg, 97)
    folder = lc.write_folder(tmp_path / "m", cfg, params)
    toks = lc.tokens(cfg, 30, 98)
    ref, _ = lc.plain(params, cfg, toks)
    r = subprocess.run([sys.executable, "-m", "camelid_b200.generate", "--model", str(folder), "--dtype", "float32", "-n", "5", "--tokens",
                        ",".join(map(str, toks)), "--tokens", "1,2"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    lines = r.stdout.strip().splitlines()
    assert len(lines) == 2
    greedy_follows(params, cfg, toks, [int(t) for t in lines[0].split(",")], "float32")
    for dtype in DTYPES:
        out = tmp_path / dtype
        out.mkdir()
        steps = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:11], "want": [0, 10]}], "end": []},
                 {"step": 1, "entries": [{"id": "x", "tokens": toks[11:13], "want": []}], "end": []},
                 {"step": 2, "entries": [{"id": "y", "tokens": toks[:3], "want": [2]}, {"id": "x", "tokens": toks[13:], "want": [1, 16]}], "end": ["x", "y"]},
                 {"step": 3, "entries": [{"id": "z", "tokens": toks[:1], "want": [0]}], "end": ["z"]}]
        r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32", "3.f32"]
        for step, places in ((0, [0, 10]), (2, [2, 14, 29]), (3, [0])):
            got = np.fromfile(out / f"{step}.f32", "<f4").reshape(-1, cfg["vocab"])
            check(got, ref[places], dtype, step)
