"""Host-side parts of the Pefolix family that need no GPU: the registry, the build's parts, checkpoints, the replay
loop, the command lines, and properties of the plain oracle itself."""
import json

import numpy as np
import pytest

from oracle import pefolix_oracle as po


def test_registry_by_architecture(tmp_path):
    from lemonade_burn_b200 import _lib, build, model, pefolix, runtime  # noqa: F401
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Pefolix"}))
    assert runtime.architecture_of(tmp_path) == "Pefolix" and runtime._FAMILIES["Pefolix"] is pefolix.NativePefolix
    (tmp_path / "config.json").write_text("{}")
    assert runtime.architecture_of(tmp_path) == "" and runtime._FAMILIES[""] is model.NativeBitNet
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nobody"}))
    with pytest.raises(ValueError, match="no model family"):
        runtime.load_model(tmp_path, ctx=object())
    with pytest.raises(ValueError, match="dtype"):
        runtime.load_model(tmp_path, ctx=object(), dtype="float16")
    build.build()
    lib = _lib.load()
    assert lib.lbk_model_has_architecture(b"Pefolix") and lib.lbk_model_has_architecture(b"") and not lib.lbk_model_has_architecture(b"Nobody")


def test_build_parts_cover_the_sources():
    """Every source is the runtime's or a family's; families may share kernel files, not each other's model file."""
    from lemonade_burn_b200 import build
    assert sorted(build.SOURCES) == sorted(p.name for p in build.CSRC.glob("*.cu"))
    assert len(build.SOURCES) == len(set(build.SOURCES))
    assert set(build.FAMILIES) == {"", "Pefolix", "Dugulorn"}
    for name, sources in build.FAMILIES.items():
        assert not any(f"lbk_{other.lower()}.cu" in sources for other in build.FAMILIES if other and other != name)
    build.build()
    assert build.library_for("Pefolix") == build.LIB   # the whole library is there and fresh


def test_checkpoint_round_trip(tmp_path):
    from lemonade_burn_b200 import pefolix as p
    cfg = p.make_config(37, 24, [p.attention_layer(3, 1, 8, 12, 5, 2, 0.3, p.moe_mlp(3, 2, 10, 6)), p.attention_layer(2, 2, 4, None, None, 0, None, None),
                                 p.attention_layer(2, 1, 4, 4, 3, 0, 0.5, p.dense_mlp(14))])
    t = p.random_checkpoint(cfg, 3)
    assert {n: v.shape for n, v in t.items()} == dict(p.tensor_shapes(cfg))
    p.save_checkpoint(tmp_path, cfg, t)
    cfg2, w = po.load(tmp_path)
    assert cfg2 == cfg and set(w) == set(t)
    for n in t:
        assert np.array_equal(w[n], p.bf16_values(t[n]).astype(np.float64))
    assert po.forward(cfg2, w, [1, 2, 3, 4]).shape == (4, 37)
    assert p.bf16_values(p.bf16_bits(np.array([1.0 + 2.0 ** -8, 1.0 + 3 * 2.0 ** -8], np.float32))).tolist() == [1.0, 1.0 + 2.0 ** -6]  # ties to even


def test_replay_loop_without_a_model(tmp_path):
    """Caches are made when a request appears, given back when it ends, and taken over by the next; a step in which
    nothing is wanted writes no file."""
    from lemonade_burn_b200 import trace

    class Net:
        made, log, ctx = 0, [], type("C", (), {"check_device_error": lambda self: None})()

        def new_cache(self, b, cap):
            Net.made += 1
            assert (b, cap) == (1, 16)
            return Net.made

        def reset_cache(self, c):
            self.log.append(("reset", c))

        def forward_rows(self, toks, c, want):
            self.log.append((c, list(toks)))
            return np.array([[toks[p], c] for p in want], dtype=np.float32).reshape(-1, 2)

    lines = ['{"step": 0, "entries": [{"id": "a", "tokens": [4, 5], "want": [1, 0]}], "end": []}', "",
             '{"step": 1, "entries": [{"id": "a", "tokens": [6], "want": []}], "end": ["a"]}',
             '{"step": 2, "entries": [{"id": "b", "tokens": [7], "want": [0]}], "end": ["b"]}']
    done = []
    trace.replay(Net(), lines, tmp_path, 16, done.append)
    assert done == [0, 1, 2] and Net.made == 1 and Net.log == [(1, [4, 5]), (1, [6]), ("reset", 1), (1, [7]), ("reset", 1)]
    assert np.fromfile(tmp_path / "0.f32", dtype="<f4").tolist() == [5, 1, 4, 1]
    assert not (tmp_path / "1.f32").exists() and np.fromfile(tmp_path / "2.f32", dtype="<f4").tolist() == [7, 1]


def test_command_lines():
    from lemonade_burn_b200 import generate, trace
    for main in (generate.main, trace.main):
        with pytest.raises(SystemExit):
            main([])
        with pytest.raises(SystemExit):
            main(["--model", "x", "--dtype", "int8", "--out", "y", "--prompt", "1"])


def test_oracle_slopes_and_visibility():
    assert np.allclose(po.slopes(8), [2.0 ** -(h + 1) for h in range(8)])
    assert np.allclose(po.slopes(12)[[2, 11]], [2.0 ** -2, 2.0 ** -8])
    see = po.visible([9], np.arange(12), {"size": 4, "keep_first": 2})[0]
    assert see.tolist() == [j < 2 or 5 < j < 10 for j in range(12)]
    assert po.visible([3], np.arange(5), None)[0].tolist() == [True] * 4 + [False]


def test_oracle_attention_by_hand():
    """Two heads on one key/value head, a window of two with one kept token, written out term by term."""
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((5, 2, 3)), rng.standard_normal((5, 1, 3)), rng.standard_normal((5, 1, 2))
    out = po.attention(q, k, v, 0.7, {"size": 2, "keep_first": 1}, np.arange(5), np.arange(5))
    for h, slope in ((0, 2.0 ** -4), (1, 2.0 ** -8)):
        e = {j: np.exp(q[4, h] @ k[j, 0] * 0.7 - slope * (4 - j)) for j in (0, 3, 4)}
        want = sum(e[j] * v[j, 0] for j in e) / sum(e.values())
        assert np.allclose(out[4, h], want)


def test_oracle_layer_norm_and_experts():
    x = np.array([[1.0, 2.0, 6.0]])
    assert np.allclose(po.layer_norm(x, np.array([1.0, 1.0, 2.0]), 0.5), (x - 3.0) / np.sqrt(14.0 / 3.0 + 0.5) * [1, 1, 2])
    ids, wt = po.route(np.eye(4)[[2]], np.diag([1.0, 2.0, 3.0, 0.0]), 2)
    s = np.exp([0.0, 0.0, 3.0, 0.0]) / (np.exp(3.0) + 3)
    assert ids.tolist() == [[2, 0]] and np.allclose(wt, s[[2, 0]])
    assert np.isclose(po.gelu_tanh(np.array(1.0)), 0.8411919906082768) and po.relu2(np.array(-2.0)) == 0.0 and po.relu2(np.array(3.0)) == 9.0
