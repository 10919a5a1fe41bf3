"""Host-side parts of the Dugulorn family that need no GPU: the registry, checkpoints, and properties of the plain oracle
itself, written out by hand."""
import json
import math

import numpy as np
import pytest

from oracle import dugulorn_oracle as do
from oracle import pefolix_oracle as po


def test_registry_by_architecture(tmp_path):
    from lemonade_burn_b200 import _lib, build, dugulorn, runtime
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Dugulorn"}))
    assert runtime.architecture_of(tmp_path) == "Dugulorn" and runtime._FAMILIES["Dugulorn"] is dugulorn.NativeDugulorn
    build.build()
    assert _lib.load().lbk_model_has_architecture(b"Dugulorn")
    assert build.library_for("Dugulorn") == build.LIB


def test_checkpoint_round_trip(tmp_path):
    from lemonade_burn_b200 import dugulorn as p
    cfg = p.make_config(37, 24, [p.lightning_layer(2, 6, 10, [0.5, 0.9], 14), p.latent_layer(3, 8, 4, 12, 9, 10, 0.3, 50.0, p.yarn(2.0, 16), None, None),
                                 p.delta_layer(4, 2, 6, 5, 3, 12), p.latent_layer(2, 6, 4, 8, 7, 10, 0.2, 50.0, None, 1, None)])
    t = p.random_checkpoint(cfg, 3, low_rank=5)
    assert {n: v.shape for n, v in t.items()} == dict(p.tensor_shapes(cfg, 5))
    assert "l3.mix.dkv" not in t and "l1.mlp.up" not in t and t["l2.mix.a1"].shape == (5, 24)
    p.save_checkpoint(tmp_path, cfg, t)
    cfg2, w = po.load(tmp_path)
    assert cfg2 == cfg and set(w) == set(t)
    out = []
    lg = do.forward(cfg2, w, [1, 2, 3, 4, 5], out)
    assert lg.shape == (5, 37) and len(out) == 4 and np.isfinite(lg).all()
    assert np.allclose(do.forward(cfg2, w, [1, 2, 3]), lg[:3])   # a decoder: the front does not know the rest


def test_rotation_by_hand():
    x = np.array([[1.0, 2.0, 3.0, 4.0]])
    y = do.rotate(x, [5], {"dims": 4, "base": 100.0})[0]
    for i, f in ((0, 1.0), (1, 0.1)):
        a = 5 * f
        assert np.allclose(y[2 * i:2 * i + 2], [x[0, 2 * i] * math.cos(a) - x[0, 2 * i + 1] * math.sin(a), x[0, 2 * i + 1] * math.cos(a) + x[0, 2 * i] * math.sin(a)])
    # scores depend on the distance only
    q, k = np.random.default_rng(0).standard_normal((2, 1, 8))
    rot = {"dims": 8, "base": 30.0}
    assert np.isclose(do.rotate(q, [9], rot)[0] @ do.rotate(k, [4], rot)[0], do.rotate(q, [109], rot)[0] @ do.rotate(k, [104], rot)[0])


def test_yarn_ends():
    """Pairs that turn often keep their frequency, pairs that hardly turn are slowed down by the factor, the ramp between."""
    sc = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}
    plain, one = do.frequencies({"dims": 64, "base": 1e4})
    f, m = do.frequencies({"dims": 64, "base": 1e4, "scaling": sc})
    turns = 4096 * plain / (2 * math.pi)
    assert one == 1.0 and np.isclose(m, 0.1 * math.log(4.0) + 1.0)
    assert np.allclose(f[turns > 40], plain[turns > 40]) and np.allclose(f[turns < 0.8], plain[turns < 0.8] / 4.0)
    ratio = f / plain
    assert (np.diff(ratio) <= 1e-12).all() and ((ratio > 0.26) & (ratio < 0.99)).sum() > 3


def test_latent_attention_by_hand():
    """Two positions, one head, written out term by term."""
    rng = np.random.default_rng(1)
    mx = {"heads": 1, "dim": 2, "rot_dim": 2, "vdim": 3, "kv_rank": 2, "scale": 0.7, "rot": {"dims": 2, "base": 10.0}}
    shapes = {"dq": (4, 5), "uq": (4, 4), "dkv": (4, 5), "uk": (2, 2), "uv": (3, 2), "g": (1, 5), "o": (5, 3)}
    w = {"m." + n: rng.standard_normal(s) for n, s in shapes.items()}
    w["m.dq.norm"], w["m.dkv.norm"] = rng.standard_normal(4), rng.standard_normal(2)
    h = rng.standard_normal((2, 5))
    lat = do.latent_kv(h, w, "m.", mx, np.arange(2), 0.1)
    y = do.latent_attention(h, w, "m.", mx, np.arange(2), 0.1, lat)
    c, kr, q, val = [], [], None, []
    for p in range(2):
        kv = w["m.dkv"] @ h[p]
        c.append(kv[:2] / math.sqrt((kv[0] ** 2 + kv[1] ** 2) / 2 + 0.1) * w["m.dkv.norm"])
        kr.append([kv[2] * math.cos(p) - kv[3] * math.sin(p), kv[3] * math.cos(p) + kv[2] * math.sin(p)])
        cq = w["m.dq"] @ h[p]
        q = w["m.uq"] @ (cq / math.sqrt((cq * cq).mean() + 0.1) * w["m.dq.norm"])
        val.append(w["m.uv"] @ c[p])
    qr = [q[2] * math.cos(1) - q[3] * math.sin(1), q[3] * math.cos(1) + q[2] * math.sin(1)]
    e = [math.exp(0.7 * (q[:2] @ (w["m.uk"] @ c[p]) + np.dot(qr, kr[p]))) for p in range(2)]
    o = (e[0] * val[0] + e[1] * val[1]) / (e[0] + e[1]) / (1 + math.exp(-float(w["m.g"][0] @ h[1])))
    assert np.allclose(y[1], w["m.o"] @ o)


def test_convolution_by_hand():
    x, taps = np.arange(1.0, 9.0).reshape(4, 2), np.array([[1.0, 10.0, 100.0], [2.0, 0.0, 5.0]])
    y = do.short_conv(x, taps)
    assert y[0].tolist() == [100.0, 10.0] and y[1].tolist() == [310.0, 20.0] and y[3].tolist() == [753.0, 48.0]


def test_recurrences_by_hand():
    rng = np.random.default_rng(2)
    q, k, v = (rng.standard_normal((3, 1, 2)) for _ in range(3))
    o = do.lightning_core(q, k, v, [0.5])
    want = sum(0.5 ** (2 - j) * (q[2, 0] @ k[j, 0]) * v[j, 0] for j in range(3))
    assert np.allclose(o[2, 0], want)
    g, beta = rng.uniform(0.2, 1.0, (3, 1, 2)), rng.uniform(0.1, 0.9, (3, 1))
    o = do.delta_core(q, k, v, g, beta)
    S = np.zeros((2, 2))
    for t in range(3):
        S = np.diag(g[t, 0]) @ S
        S = S + beta[t, 0] * np.outer(k[t, 0], v[t, 0] - S.T @ k[t, 0])
        assert np.allclose(o[t, 0], S.T @ q[t, 0])


def test_activations_and_norms():
    assert np.isclose(do.softplus(np.array(0.0)), math.log(2.0)) and np.isclose(do.softplus(np.array(50.0)), 50.0) and do.softplus(np.array(-800.0)) == 0.0
    assert do.relu2(np.array(-2.0)) == 0.0 and do.relu2(np.array(3.0)) == 9.0 and np.isclose(do.silu(np.array(1.0)), 1 / (1 + math.exp(-1)))
    assert np.allclose(do.rms_norm(np.array([3.0, 4.0]), np.array([1.0, 2.0]), 0.5), np.array([3.0, 8.0]) / math.sqrt(13.0))
    assert np.allclose(do.unit(np.array([[3.0, 4.0]])), np.array([[0.6, 0.8]]), atol=1e-6)


@pytest.mark.parametrize("kind", ["mixed", "latent", "lightning", "delta"])
def test_bench_configurations(kind):
    import bench_dugulorn as b
    from lemonade_burn_b200 import dugulorn as p
    for name in b.MODELS:
        cfg = b.config(p, name, kind)
        assert len(cfg["layers"]) == b.MODELS[name][4] and b.step_bytes(cfg, p, 16) > b.step_bytes(cfg, p, 1) > 0
        for i, layer in enumerate(cfg["layers"]):
            src = layer["mixer"].get("kv_from")
            assert src is None or (src < i and "kv_from" not in cfg["layers"][src]["mixer"])
