"""Tokovik without a GPU: the plain evaluation's own mechanisms, configuration, registry."""
import json

import numpy as np
import pytest

import layered_helpers as lh
import plain_tokovik as pt
import tokovik_cases as tc


# ---------------------------------------------------------------- the plain evaluation

def test_recurrence_equals_its_quadratic_form():
    rng = np.random.default_rng(1)
    q, k, v, a = rng.standard_normal((20, 2, 5)), rng.standard_normal((20, 2, 5)), rng.standard_normal((20, 2, 7)), rng.uniform(0.3, 1.0, (20, 2, 5))
    o = pt.gated_recurrence(q, k, v, a)
    for h in range(2):
        for t in range(20):
            want = sum((q[t, h] * np.prod(a[s + 1:t + 1, h], 0)) @ k[s, h] * v[s, h] for s in range(t + 1))
            assert np.allclose(o[t, h], want)


def test_window_has_its_own_token_and_the_ones_before_it():
    rng = np.random.default_rng(2)
    q, k, v = rng.standard_normal((9, 4, 3)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 5))
    o = pt.window_attention(q, k, v, 0.7, 4)
    for h in range(4):
        for i in range(9):
            lo = max(0, i - 3)
            p = np.exp(0.7 * k[lo:i + 1, h // 2] @ q[i, h])
            assert np.allclose(o[i, h], p @ v[lo:i + 1, h // 2] / p.sum())
    assert np.allclose(pt.window_attention(q, k, v, 0.7, 1), np.repeat(v, 2, 1))


def test_rotation_pairs_halves_keeps_scores_relative_and_passes_the_rest():
    rot = {"base": 50.0, "dims": 6, "scaling": None}
    rng = np.random.default_rng(3)
    q, k = rng.standard_normal((1, 10)), rng.standard_normal((1, 10))

    def at(x, p):
        return pt.rotated_halves(x, [p], rot)

    assert np.allclose(at(q, 9) @ at(k, 4).T, at(q, 25) @ at(k, 20).T, atol=1e-5)
    assert np.array_equal(at(q, 9)[:, 6:], q[:, 6:]) and np.allclose(at(q, 0), q)
    a = np.float32(3.0)
    assert np.allclose(at(q, 3)[0, 0], q[0, 0] * np.cos(a) - q[0, 3] * np.sin(a)) and np.allclose(at(q, 3)[0, 3], q[0, 3] * np.cos(a) + q[0, 0] * np.sin(a))


def test_yarn_keeps_fast_pairs_and_slows_the_others():
    rot = {"base": 10000.0, "dims": 64, "scaling": {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}
    f, gain = pt.yarn_frequencies(rot)
    raw = [10000.0 ** (-2.0 * i / 64) for i in range(32)]
    turns = [4096 * r / (2 * np.pi) for r in raw]
    assert all(a == r for a, r, t in zip(f, raw, turns) if t > 40) and all(np.isclose(a, r / 8) for a, r, t in zip(f, raw, turns) if t < 0.7)
    assert any(r / 8 < a * 0.999 and a < r * 0.999 for a, r in zip(f, raw)) and np.isclose(gain, 1 + 0.1 * np.log(8.0))


def test_parallel_is_half_the_sum_of_two_normed_results():
    cfg = tc.CASES["one_layer"]
    p = {k: v.astype(np.float64) for k, v in tc.random_params(cfg, 4).items()}
    w, m = pt.under(p, "l0.mix."), cfg["layers"][0]["mixer"]
    h = np.random.default_rng(5).standard_normal((6, 72))
    both = pt.parallel(h, w, m, 1e-5)
    one = pt.parallel(h, dict(w, **{"right.out": np.zeros(72)}), m, 1e-5)
    two = pt.parallel(h, dict(w, **{"left.out": np.zeros(72)}), m, 1e-5)
    assert np.allclose(both, one + two)
    assert np.allclose(((2 * one / w["left.out"]) ** 2).mean(-1), 1.0, atol=1e-3)


# ---------------------------------------------------------------- configuration, registry, files

@pytest.mark.parametrize("case", sorted(tc.CASES))
def test_spec_follows_the_configuration(case):
    from camelid_b200.layered import PARALLEL, POST_NORM, SWIGLU

    cfg = tc.CASES[case]
    s = tc.spec(json.loads(json.dumps(cfg)))
    assert (s.vocab, s.width, s.eps, s.embed_scale, s.logit_scale, s.residual, s.streams) == (
        cfg["vocab"], cfg["width"], cfg["norm"]["eps"], cfg["embedding"]["scale"], cfg["logit_scale"], POST_NORM, 1)
    assert s.runs == list(range(len(cfg["layers"])))
    for i, (got, e) in enumerate(zip(s.layers, cfg["layers"])):
        l, r, w, g = e["mixer"]["left"], e["mixer"]["right"], got.window, got.gated
        assert got.type == PARALLEL and got.mlp == SWIGLU and got.ff == (e["mlp"]["ff"] if e["mlp"] else 0)
        assert (w.heads, w.kv_heads, w.dim, w.vdim, w.window, w.scale) == (l["heads"], l["kv_heads"], l["dim"], l["vdim"], l["mask"]["size"], l["scale"])
        assert (w.rot_dims, w.rot_base) == (l["rot"]["dims"], l["rot"]["base"])
        y = l["rot"]["scaling"]
        assert (w.rot_factor, w.rot_original, w.rot_fast, w.rot_slow) == ((0, 0, 0, 0) if y is None else (y["factor"], y["original"], y["fast"], y["slow"]))
        assert (g.heads, g.dim, g.vdim, g.rank, g.tau) == (r["heads"], r["dim"], r["vdim"], cfg["ranks"][i], r["tau"])


def test_what_the_design_does_not_have_is_refused():
    first = lambda c: c["layers"][0]  # noqa: E731
    for change in (lambda c: first(c).update(type="softmax"), lambda c: first(c).update(mlp={"kind": "moe", "ff": 3}),
                   lambda c: first(c)["mixer"]["left"].update(kv_heads=4), lambda c: first(c)["mixer"]["left"]["mask"].update(size=0),
                   lambda c: first(c)["mixer"]["left"]["rot"].update(dims=26), lambda c: first(c)["mixer"]["left"]["rot"].update(dims=3)):
        cfg = json.loads(json.dumps(tc.CASES["one_layer"]))
        change(cfg)
        with pytest.raises(ValueError):
            tc.spec(cfg)


def test_registry_picks_by_config(tmp_path):
    from camelid_b200 import models

    cfg = tc.CASES["one_layer"]
    folder = lh.write_folder(tmp_path / "m", cfg, tc.random_params(cfg, 1))
    assert models.architecture_of(folder) == "Tokovik" and "Tokovik" in models.ARCHITECTURES
    with pytest.raises(ValueError, match="max_pos"):
        models.load_model(folder)


def test_no_device_is_an_error(cm):
    if cm.device_count() > 0:
        pytest.skip("a CUDA device is present")
    cfg = tc.CASES["one_layer"]
    with pytest.raises(cm.CmldError, match="no CPU path"):
        tc.engine(cfg, tc.random_params(cfg, 1), 16)


def test_sizes_and_constants_are_checked_before_the_device(cm):
    from camelid_b200.layered import LayeredEngine

    for change, code in ((lambda s: setattr(s, "streams", 2), 1), (lambda s: setattr(s.layers[0].gated, "tau", 0.0), 1),
                         (lambda s: setattr(s.layers[0].window, "kv_heads", 5), 2), (lambda s: setattr(s.layers[0].gated, "dim", 600), 2),
                         (lambda s: setattr(s.layers[0].window, "rot_fast", 0.0), 1), (lambda s: setattr(s, "residual", 0), 3)):
        s = tc.spec(tc.CASES["one_layer"])
        change(s)
        with pytest.raises(cm.CmldError) as e:
            LayeredEngine(s, 16)
        assert e.value.code == code
