"""Gofilorn without a GPU: the plain restatement's mechanisms against formulas
written out, the reading of config.json and of safetensors files, and the layout
that the kernels read, multiplied out."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import gofilorn as plain
from tests import gofilorn_models as models_of
from vx_b200 import gofilorn, models, safetensors, trace

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
rng = np.random.default_rng(5)


def test_norm_gain_is_one_plus_its_weight():
    x, w = rng.standard_normal((3, 10)), rng.standard_normal(10)
    got = plain.rms_norm(x, w, 0.25)
    for t in range(3):
        rms = np.sqrt(np.mean(x[t] ** 2) + 0.25)
        assert np.allclose(got[t], x[t] / rms + w * x[t] / rms)


def test_position_vector_interleaves_sine_and_cosine():
    v = plain.position_vector(9, 6)
    f = [1.0, 10000.0 ** (-1 / 3), 10000.0 ** (-2 / 3)]
    assert np.allclose(v[0::2], np.sin([9 * a for a in f]))
    assert np.allclose(v[1::2], np.cos([9 * a for a in f]))


def test_window_of_one_returns_the_own_key_and_softmax_weighs_two():
    q, k = rng.standard_normal((4, 2, 3)), rng.standard_normal((4, 1, 3))
    alone = plain.attention(q, k, 1, 0.7)
    assert np.allclose(alone, np.repeat(k, 2, axis=1))
    two = plain.attention(q, k, 2, 0.7)
    s = [0.7 * q[3, 1] @ k[2, 0], 0.7 * q[3, 1] @ k[3, 0]]
    p = 1.0 / (1.0 + np.exp(s[1] - s[0]))
    assert np.allclose(two[3, 1], p * k[2, 0] + (1 - p) * k[3, 0])


@pytest.mark.parametrize("name", sorted(models_of.CONFIGS))
def test_a_prefix_has_the_same_logits(name):
    cfg = models_of.CONFIGS[name]
    w = models_of.weights(cfg)
    tokens = rng.integers(0, cfg["vocab"], 24)
    whole = plain.logits(tokens, w, cfg)
    part = plain.logits(tokens[:17], w, cfg)
    assert np.allclose(whole[:17], part)


def test_the_marked_token_shows_a_window_that_is_one_off():
    """The inputs of the window tests on the GPU: an oracle whose window is one
    position too long or too short gives clearly other logits at the edge."""
    cfg, w, token = models_of.marked(16)
    tokens = rng.integers(0, cfg["vocab"] - 1, 40)
    tokens[8] = token
    right = plain.logits(tokens, w, cfg)
    scale = np.sqrt(np.mean(right ** 2))
    for wrong, at in ((15, 8 + 15), (17, 8 + 16)):
        off = copy.deepcopy(cfg)
        off["layers"][0]["mixer"]["mask"]["size"] = wrong
        bad = plain.logits(tokens, w, off)
        assert np.sqrt(np.mean((bad[at] - right[at]) ** 2)) > 0.02 * scale
        assert np.allclose(bad[:at], right[:at])


@pytest.mark.parametrize("name", sorted(models_of.CONFIGS))
def test_packed_matrices_multiply_out_to_the_layer(name):
    """q | k | gate | up and attention | up with their filling, against the plain
    layer."""
    cfg = models_of.CONFIGS[name]
    w = models_of.weights(cfg, seed=3)
    parsed = gofilorn.GofilornConfig.from_dict(cfg)
    assert parsed.dim % 64 == 0 and parsed.vocab_rows % 8 == 0
    x = rng.standard_normal((6, cfg["width"]))
    for i, s in enumerate(parsed.layers):
        n = "l%d." % s.source
        assert s.source == plain.owner(cfg["layers"], i)
        w_in, w_out = gofilorn.pack_layer(
            s, cfg["width"], parsed.dim,
            lambda name, shape: models_of.getter(w)(n + name, shape))
        assert w_in.shape == (s.in_rows, parsed.dim)
        assert w_out.shape == (parsed.dim, s.out_cols) and s.out_cols % 64 == 0
        gain = gofilorn.pack_gain(w[n + "norm1"], parsed.dim)
        full = np.zeros((6, parsed.dim))
        full[:, :cfg["width"]] = x
        inv = 1.0 / np.sqrt((full ** 2).sum(1, keepdims=True) / cfg["width"]
                            + parsed.eps)
        y = (full * inv * gain) @ w_in.astype(np.float64).T
        P, att, kv = s.head_dim, s.att, s.kv_heads * s.head_dim
        q = y[:, :att].reshape(6, s.heads, P)
        k = y[:, att:att + kv].reshape(6, s.kv_heads, P)
        g = 1.0 / (1.0 + np.exp(-y[:, att + kv:2 * att + kv]))
        u = np.maximum(y[:, 2 * att + kv:], 0.0) ** 2
        a = plain.attention(q, k, s.window, s.scale).reshape(6, att) * g
        out = full + np.concatenate([a, u], axis=1) @ w_out.astype(np.float64).T
        want = plain.layer(x, w, cfg, i)
        assert np.abs(out[:, :cfg["width"]] - want).max() < 1e-5 * np.abs(want).max()
        assert not out[:, cfg["width"]:].any()


def test_turns_are_the_angles_of_the_position_vector():
    for width in (6, 77, 128):
        turns = gofilorn.turns_per_position(width)
        for p in (0, 1, 5000, 123457):
            v = plain.position_vector(p, width)
            i = np.arange(width) // 2
            angle = 2 * np.pi * np.mod(p * turns[i], 1.0)
            mine = np.where(np.arange(width) % 2 == 0, np.sin(angle), np.cos(angle))
            assert np.abs(mine - v).max() < 1e-9


def test_what_a_configuration_may_not_say():
    def broken(change):
        cfg = copy.deepcopy(models_of.UNEVEN)
        change(cfg)
        with pytest.raises(ValueError):
            gofilorn.GofilornConfig.from_dict(cfg)
    broken(lambda c: c.update(architecture="other"))
    broken(lambda c: c["layers"][0].update(type="recurrent"))
    broken(lambda c: c["layers"][0]["mixer"].update(vdim=16))
    broken(lambda c: c["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="experts"))
    broken(lambda c: c["layers"][3].update(weights_of=9))
    broken(lambda c: c["layers"][3].update(weights_of=1))      # other sizes
    broken(lambda c: c["layers"][0].update(weights_of=3))      # nobody has tensors


def test_tensors_by_way_of_a_layer_that_borrows_them():
    cfg = copy.deepcopy(models_of.EVEN)
    cfg["layers"].append(dict(cfg["layers"][0], weights_of=2))
    parsed = gofilorn.GofilornConfig.from_dict(cfg)
    assert [s.source for s in parsed.layers] == [0, 1, 0, 0]
    assert plain.owner(cfg["layers"], 3) == 0


def test_safetensors_file(tmp_path):
    cfg = models_of.ODD_WIDTH
    w = models_of.weights(cfg)
    models_of.write(str(tmp_path), cfg, w)
    f = safetensors.SafeTensors(str(tmp_path / "model.safetensors"))
    assert sorted(f.names()) == sorted(w)
    for name, a in w.items():
        assert np.array_equal(f.f32(name, a.shape), a.astype(np.float32))
        assert np.array_equal((safetensors.to_bf16(a).astype(np.uint32) << 16)
                              .view(np.float32), a.astype(np.float32))
    with pytest.raises(ValueError):
        f.f32("embed", (1, 2))
    with pytest.raises(ValueError):
        f.f32("absent")
    short = tmp_path / "short"
    short.write_bytes(b"abc")
    with pytest.raises(ValueError):
        safetensors.SafeTensors(str(short))


def test_the_registry_goes_by_config_json(tmp_path):
    models_of.write(str(tmp_path), models_of.ODD_WIDTH, {})
    assert models.architecture_of(str(tmp_path)) == "Gofilorn"
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nobody"}))
    with pytest.raises(ValueError):
        models.load(str(tmp_path))
    with pytest.raises(models.UnsupportedDtype):
        models.load(str(tmp_path / "weights.bin"), "bfloat16")


class FakeDecoder:
    """Counts what it is fed; its logits are (position, token)."""

    def __init__(self):
        self.pos, self.resets = 0, 0

    def reset(self):
        self.pos, self.resets = 0, self.resets + 1

    def feed(self, tokens, want=()):
        rows = [[self.pos + i, t] for i, t in enumerate(tokens) if i in want]
        self.pos += len(tokens)
        return np.array(rows, np.float32).reshape(len(want), 2)


def test_replay_keeps_the_order_of_the_wanted_places_and_the_requests_apart():
    d = FakeDecoder()
    r = trace.Replay(d)
    rows = r.step([{"id": "a", "tokens": [5, 6, 7], "want": [2, 0]}], [])
    assert np.concatenate(rows).tolist() == [[2, 7], [0, 5]]
    assert r.step([{"id": "a", "tokens": [8], "want": []}], ["a"]) == []
    rows = r.step([{"id": "b", "tokens": [9], "want": [0]}], [])
    assert rows[0].tolist() == [[0, 9]] and d.resets == 2
    with pytest.raises(ValueError):
        r.step([{"id": "c", "tokens": [1], "want": []}], [])
    with pytest.raises(ValueError):
        r.step([{"id": "b", "tokens": [1], "want": [1]}], [])


def test_a_model_that_does_not_run_in_the_number_format_ends_with_3(tmp_path):
    (tmp_path / "weights.bin").write_bytes(b"\0" * 64)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"),
                        "--model", str(tmp_path / "weights.bin"), "--dtype",
                        "bfloat16", "--out", str(tmp_path)], input="", text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 3, r.stderr
