"""Losarax without a GPU: the plain evaluation's own mechanisms, configuration, registry, checkpoint files, scheduler and
trace replay on a stand-in engine."""
import json

import numpy as np
import pytest

import losarax_cases as lc
import plain_losarax as pl


# ---------------------------------------------------------------- the plain evaluation

def test_recurrence_equals_its_quadratic_form():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((20, 2, 5)), rng.standard_normal((20, 2, 5)), rng.standard_normal((20, 2, 7))
    decay = [0.6, 0.99]
    o = pl.decayed_outer_product_recurrence(q, k, v, decay)
    i, j = np.arange(20)[:, None], np.arange(20)[None, :]
    for h in range(2):
        w = np.where(j <= i, decay[h] ** np.maximum(i - j, 0), 0.0) * (q[:, h] @ k[:, h].T)
        assert np.allclose(o[:, h], w @ v[:, h])


def test_rotation_keeps_scores_relative_and_passes_the_rest():
    rng = np.random.default_rng(2)
    q, k = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))

    def at(x, p):
        return pl.rotate_interleaved(x, [p], 6, 50.0)

    assert np.allclose(at(q, 9) @ at(k, 4).T, at(q, 25) @ at(k, 20).T, atol=1e-5)
    assert np.array_equal(at(q, 9)[:, 6:], q[:, 6:]) and np.allclose(at(q, 0), q)
    a = np.float32(3.0)
    assert np.allclose(at(q, 3)[0, 0], q[0, 0] * np.cos(a) - q[0, 1] * np.sin(a)) and np.allclose(at(q, 3)[0, 1], q[0, 1] * np.cos(a) + q[0, 0] * np.sin(a))


def test_attention_sees_no_later_key_and_itself():
    rng = np.random.default_rng(3)
    q, k, v = (rng.standard_normal((6, 2, 4)) for _ in range(3))
    o = pl.causal_softmax_attention(q, k, v, 0.5)
    assert np.allclose(o[0], v[0])
    k2, v2 = k.copy(), v.copy()
    k2[4:], v2[4:] = 9.0, 9.0
    o2 = pl.causal_softmax_attention(q, k2, v2, 0.5)
    assert np.allclose(o[:4], o2[:4]) and not np.allclose(o[4], o2[4])


def test_hyper_connection_mixes_from_rows_to_columns():
    xs = np.arange(12.0).reshape(3, 2, 2)
    w = {"in": np.array([0.0, 2.0, 0.0]), "out": np.array([1.0, 0.0, -1.0]), "mix": np.zeros((3, 3))}
    w["mix"][0, 2] = 5.0  # stream 0 goes to stream 2
    out = pl.hyper_connection(xs, w, lambda u: u, lambda u: u + 1)
    assert np.allclose(out[0], 2 * xs[1] + 1) and np.allclose(out[1], 0) and np.allclose(out[2], 5 * xs[0] - 2 * xs[1] - 1)


def test_layer_order_of_loops():
    cfg = lc.config([lc.lightning()] * 4, loop={"start": 1, "stop": 3, "times": 3})
    assert pl.layer_order(cfg) == [0, 1, 2, 1, 2, 1, 2, 3]


# ---------------------------------------------------------------- configuration, registry, files

@pytest.mark.parametrize("case", sorted(lc.CASES))
def test_spec_follows_the_configuration(case):
    from camelid_b200 import losarax
    from camelid_b200.layered import LATENT

    cfg = lc.CASES[case]
    spec = losarax.spec_from_config(json.loads(json.dumps(cfg)))
    assert spec.runs == pl.layer_order(cfg) and spec.streams == cfg["streams"] and spec.eps == cfg["norm"]["eps"]
    for s, layer in zip(spec.layers, cfg["layers"]):
        m = layer["mixer"]
        assert (s.heads, s.dim, s.vdim) == (m["heads"], m["dim"], m["vdim"])
        assert s.ff == (layer["mlp"]["ff"] if layer["mlp"] else 0)
        if s.type == LATENT:
            assert (s.q_rank, s.kv_rank, s.rot_dim, s.rot_dims, s.rot_base, s.scale) == (m["q_rank"], m["kv_rank"], m["rot_dim"], m["rot"]["dims"],
                                                                                         m["rot"]["base"], m["scale"])
        else:
            assert s.decay == m["decay"]


def test_what_the_design_does_not_have_is_refused():
    from camelid_b200 import losarax

    for change in (lambda c: c["layers"][0].update(type="softmax"), lambda c: c["layers"][0].update(mlp={"kind": "moe", "ff": 3}),
                   lambda c: c["layers"][0]["mixer"].update(decay=[0.5]), lambda c: c.update(loop={"start": 0, "stop": 5, "times": 2})):
        cfg = json.loads(json.dumps(lc.CASES["lightning"]))
        change(cfg)
        with pytest.raises(ValueError):
            losarax.spec_from_config(cfg)


def test_registry_picks_by_config_and_metadata(tmp_path):
    from camelid_b200 import gguf, models

    cfg = lc.CASES["latent"]
    folder = lc.write_folder(tmp_path / "m", cfg, lc.random_params(cfg, 1))
    assert models.architecture_of(folder) == "Losarax"
    gguf.write_gguf(tmp_path / "x.gguf", {"general.architecture": "llama"}, [("t", gguf.F32, (4,), np.zeros(4, np.float32).view(np.uint8))])
    assert models.architecture_of(tmp_path / "x.gguf") == "llama" and "llama" in models.ARCHITECTURES
    (tmp_path / "y").mkdir()
    (tmp_path / "y" / "config.json").write_text('{"architecture": "unheard-of"}')
    with pytest.raises(ValueError, match="unheard-of"):
        models.load_model(tmp_path / "y", max_pos=8)
    with pytest.raises(ValueError, match="max_pos"):
        models.load_model(folder)


def test_no_device_is_an_error_for_layered_engines(cm):
    if cm.device_count() > 0:
        pytest.skip("a CUDA device is present")
    cfg = lc.CASES["latent"]
    with pytest.raises(cm.CmldError, match="no CPU path"):
        lc.engine(cfg, lc.random_params(cfg, 1), 16)


def test_safetensors_round_trip(tmp_path):
    from camelid_b200.safetensors import SafetensorsFile, from_bf16, to_bf16, write_safetensors

    x = np.random.default_rng(0).standard_normal((3, 5)).astype(np.float32)
    write_safetensors(tmp_path / "a.safetensors", {"w": to_bf16(x).reshape(3, 5), "t": np.arange(4, dtype=np.int32)})
    f = SafetensorsFile(tmp_path / "a.safetensors")
    assert f.shape("w") == (3, 5) and f.dtype("w") == "BF16" and f.dtype("t") == "I32"
    assert np.array_equal(f.data("t"), np.arange(4)) and np.allclose(from_bf16(f.data("w")), x, rtol=2 ** -8)
    f.close()
    (tmp_path / "bad.safetensors").write_bytes(b"\xff" * 40)
    with pytest.raises(ValueError):
        SafetensorsFile(tmp_path / "bad.safetensors")
    data = (tmp_path / "a.safetensors").read_bytes()
    (tmp_path / "short.safetensors").write_bytes(data[:-3])
    with pytest.raises(ValueError, match="outside the file"):
        SafetensorsFile(tmp_path / "short.safetensors")


def test_bf16_rounds_to_nearest_even():
    from camelid_b200.safetensors import from_bf16, to_bf16

    x = np.array([1.0, 1.0 + 2.0 ** -8, 1.0 + 3 * 2.0 ** -8, -2.5, 1.0 + 2.0 ** -8 + 2.0 ** -20], np.float32)
    assert from_bf16(to_bf16(x)).tolist() == [1.0, 1.0, 1.0 + 2.0 ** -6, -2.5, 1.0 + 2.0 ** -7]


# ---------------------------------------------------------------- scheduler and trace replay on a stand-in engine

class StandIn:
    """An engine whose next token is a function of everything its slot has seen, and which checks the slot discipline."""

    def __init__(self, max_seqs, max_pos=64, vocab=97):
        from camelid_b200.layered import LayeredRuntime

        self.cfg = LayeredRuntime(vocab, 4, max_pos, max_seqs)
        self.seen = {}
        self.calls = []

    def _feed(self, seq, tokens, pos):
        if pos == 0:
            self.seen[seq] = []
        assert len(self.seen.get(seq, [])) == pos, "a slot continues where it ends"
        self.seen[seq] = self.seen[seq] + [int(t) for t in tokens]
        return self.value(self.seen[seq])

    def value(self, toks):
        return sum((i + 3) * t for i, t in enumerate(toks)) % self.cfg.vocab

    def extend(self, seq, tokens, start_pos, want=(), taps=0):
        self.calls.append(("extend", seq, len(tokens)))
        logits = []
        for i, t in enumerate(tokens):
            nxt = self._feed(seq, [t], start_pos + i)
            if i in want:
                logits.append([nxt, len(self.seen[seq]), seq, t])
        self.last = {-1: nxt}
        return nxt, np.array(logits, np.float32).reshape(len(want), 4)

    def step_batch(self, seqs, toks, pos):
        assert len(set(seqs)) == len(seqs)
        self.calls.append(("step", tuple(seqs)))
        out = [self._feed(s, [t], p) for s, t, p in zip(seqs, toks, pos)]
        self.last = dict(enumerate(out))
        return np.array(out), None, None

    def decode_greedy(self, seqs, toks, pos, n):
        self.calls.append(("greedy", tuple(seqs), n))
        out, cur = [], list(toks)
        for i in range(n):
            cur = [self._feed(s, [t], p + i) for s, t, p in zip(seqs, cur, pos)]
            out.append(cur)
        return np.array(out)

    def sample(self, temperature, seed, min_p=0.0, row=-1):
        return (self.last[row] + seed) % self.cfg.vocab


def alone(engine, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(engine.value(toks))
    return toks[len(prompt):]


@pytest.mark.parametrize("portion", [0, 1, 3])
def test_scheduler_serves_more_requests_than_slots(portion):
    from camelid_b200.scheduler import Scheduler

    eng = StandIn(max_seqs=2)
    s = Scheduler(eng, portion=portion)
    rng = np.random.default_rng(5)
    prompts = {f"r{i}": rng.integers(0, 97, n).tolist() for i, n in enumerate((5, 1, 9, 2, 7))}
    for i, (rid, p) in enumerate(prompts.items()):
        s.submit(rid, p, 3 + 4 * i)
    out = s.run()
    assert {r: len(t) for r, t in out.items()} == {f"r{i}": 3 + 4 * i for i in range(5)}
    for rid, p in prompts.items():
        assert out[rid] == alone(eng, p, len(out[rid]))
    assert any(c[0] == "step" and len(c[1]) == 2 for c in eng.calls) and any(c[0] == "greedy" for c in eng.calls)
    assert len(s.slots) == 0 and s.slots.free == 2


def test_scheduler_samples_and_stops():
    from camelid_b200.scheduler import Scheduler

    eng = StandIn(max_seqs=2)
    s = Scheduler(eng)
    stop_at = alone(eng, [4, 5], 6)[3]
    s.submit("a", [1, 2, 3], 4, temperature=0.7, seed=11)
    s.submit("b", [4, 5], 30, stop=[stop_at])
    out = s.run()
    toks = [1, 2, 3]
    for i in range(4):
        toks.append((eng.value(toks) + 11 + i) % 97)
    assert out["a"] == toks[3:]
    first = alone(eng, [4, 5], 6).index(stop_at)
    assert out["b"] == alone(eng, [4, 5], first + 1)
    with pytest.raises(ValueError, match="exceed"):
        s.submit("c", [1] * 60, 9)


def test_slot_table_refuses_a_request_too_many():
    from camelid_b200.scheduler import SlotTable

    t = SlotTable(1)
    t.acquire("a")
    with pytest.raises(RuntimeError, match="no free slot"):
        t.acquire("b")
    t.release("a")
    assert t.acquire("b") == 0 and t.length("b") == 0


def test_trace_replay_keeps_requests_apart_and_orders_places():
    from camelid_b200.trace import TraceRunner

    eng = StandIn(max_seqs=2)
    r = TraceRunner(eng)
    assert r.step([{"id": "a", "tokens": [1, 2, 3], "want": []}], []) is None
    got = r.step([{"id": "b", "tokens": [7, 8], "want": [1, 0]}, {"id": "a", "tokens": [4], "want": [0]}], ["b"])
    assert got[:, 1].tolist() == [2, 1, 4] and got[:, 3].tolist() == [8, 7, 4]
    got = r.step([{"id": "c", "tokens": [9], "want": [0]}], ["a", "c"])  # takes b's slot
    assert got[0].tolist() == [eng.value([9]), 1, 1, 9]
    assert len(r.slots) == 0
