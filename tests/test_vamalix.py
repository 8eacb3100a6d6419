"""Vamalix without a GPU: the plain restatement's mechanisms against formulas written
out, the reading of config.json, and the layout that the kernels read, multiplied
out the way they do it."""
import copy
import json
import math

import numpy as np
import pytest

from oracle import vamalix as plain
from tests import vamalix_models as models_of
from vx_b200 import models, safetensors, vamalix
from vx_b200.lib import MIXER_LATENT

rng = np.random.default_rng(15)


def test_rotation_turns_neighbouring_pairs_and_scores_see_distances():
    x, y = rng.standard_normal(6), rng.standard_normal(6)
    assert np.allclose(plain.rotate(x, 0, 100.0), x)
    turned = plain.rotate(x, 5, 100.0)
    for i in range(3):
        z = complex(x[2 * i], x[2 * i + 1]) * np.exp(1j * 5 * 100.0 ** (-2 * i / 6))
        assert np.allclose(turned[2 * i:2 * i + 2], [z.real, z.imag])
    near = plain.rotate(x, 9, 100.0) @ plain.rotate(y, 7, 100.0)
    far = plain.rotate(x, 1009, 100.0) @ plain.rotate(y, 1007, 100.0)
    assert np.allclose(near, far) and not np.allclose(near, x @ y)


def test_norm_gelu_and_decay():
    x, w = rng.standard_normal((2, 5)), rng.standard_normal(5)
    got = plain.rms_norm(x, w, 0.3)
    assert np.allclose(got[1], w * x[1] / math.sqrt(np.mean(x[1] ** 2) + 0.3))
    z = np.array([-9.0, -1.3, 0.0, 0.4, 5.0])
    assert np.allclose(plain.gelu(z), [0.5 * v * (1 + math.erf(v / math.sqrt(2)))
                                       for v in z], atol=1e-15)
    cfg = models_of.config(8, 5, [models_of.linear(2, 3, 4, 5.0, 2)])
    w = models_of.weights(cfg)
    h = rng.standard_normal((3, 8))
    a = plain.decays(h, w, "l0", 5.0)
    z = h @ (w["l0.mix.a2"] @ w["l0.mix.a1"]).T + w["l0.mix.a2.b"]
    assert np.allclose(a, (1.0 / (1.0 + np.exp(-z))) ** 0.2)


def test_recurrence_is_a_sum_over_all_earlier_positions():
    q, k = rng.standard_normal((6, 3)), rng.standard_normal((6, 3))
    v, a = rng.standard_normal((6, 4)), rng.uniform(0.2, 1.0, (6, 3))
    o, state = plain.recurrence(q, k, v, a)
    for i in range(6):
        want = np.zeros(4)
        for j in range(i + 1):
            want += (q[i] * np.prod(a[j + 1:i + 1], axis=0)) @ k[j] * v[j]
        assert np.allclose(o[i], want)
    head, mid = plain.recurrence(q[:2], k[:2], v[:2], a[:2])
    rest, end = plain.recurrence(q[2:], k[2:], v[2:], a[2:], mid)
    assert np.allclose(np.concatenate([head, rest]), o) and np.allclose(end, state)


def test_streams_mix_from_the_first_index_to_the_second():
    x, y = rng.standard_normal((2, 3, 4)), rng.standard_normal((3, 4))
    mix, out = np.array([[1.0, 2.0], [3.0, 4.0]]), np.array([5.0, 6.0])
    new = plain.mixed_streams(x, y, mix, out)
    assert np.allclose(new[0], 1 * x[0] + 3 * x[1] + 5 * y)
    assert np.allclose(new[1], 2 * x[0] + 4 * x[1] + 6 * y)


def test_one_stream_of_ones_is_the_ordinary_residual():
    cfg = models_of.SMALL
    w = models_of.weights(cfg)
    for name in w:
        if ".hc" in name:
            w[name] = np.ones_like(w[name])
    x = rng.standard_normal((1, 5, cfg["width"]))
    eps = cfg["norm"]["eps"]
    new = plain.layer(x, 0, w, cfg, 1)[0]
    mid = x[0] + plain.latent_attention(plain.rms_norm(x[0], w["l1.norm1"], eps), 0, w,
                                        "l1", cfg["layers"][1]["mixer"], eps)
    want = mid + plain.feed_forward(plain.rms_norm(mid, w["l1.norm2"], eps), w, "l1")
    assert np.allclose(new, want)


def test_layers_run_in_the_order_of_the_loop():
    cfg = models_of.config(8, 5, [models_of.linear(1, 3, 4, 5.0, 2)] * 5)
    assert plain.order(cfg) == [0, 1, 2, 3, 4]
    for loop, want in (((1, 3, 3), [0, 1, 2, 1, 2, 1, 2, 3, 4]),
                       ((0, 5, 2), [0, 1, 2, 3, 4] * 2), ((4, 5, 1), [0, 1, 2, 3, 4]),
                       ((0, 1, 4), [0, 0, 0, 0, 1, 2, 3, 4])):
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
        assert plain.order(cfg) == want
        assert vamalix.VamalixConfig.from_dict(cfg).order == want


@pytest.mark.parametrize("name", sorted(models_of.CONFIGS))
def test_a_prefix_has_the_same_logits(name):
    cfg = models_of.CONFIGS[name]
    w = models_of.weights(cfg)
    tokens = rng.integers(0, cfg["vocab"], 24)
    assert np.allclose(plain.logits(tokens, w, cfg)[:17],
                       plain.logits(tokens[:17], w, cfg))


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
        assert np.sqrt(np.mean((bad[at] - right[at]) ** 2)) > 0.1 * scale
        assert np.allclose(bad[:at], right[:at])


def test_a_state_that_is_lost_shows():
    """The same for the recurrence: begun afresh somewhere, the slow decays of the
    far-memory model give clearly other logits long after."""
    cfg, w = models_of.slow_decays()
    tokens = rng.integers(0, cfg["vocab"], 120)
    right = plain.logits(tokens, w, cfg)
    bad = plain.logits(tokens[20:], w, cfg)
    err = np.sqrt(np.mean((bad[-1] - right[-1]) ** 2) / np.mean(right[-1] ** 2))
    assert err > 0.02


def packed_latent(p, s, h, first):
    """A latent layer's mixer from the packed arrays, the way a step computes it:
    queries for the latents, a softmax over latents, values out of their sum."""
    T = h.shape[0]
    K, R, H = s.kv_rank, s.rot_dim, s.heads
    down = h @ p["w_in"].astype(np.float64).T

    def normed(x, gain, mean):
        return x / np.sqrt((x * x).sum(1, keepdims=True) / mean + 1e-4) * gain

    q = normed(down[:, :s.q_rank], p["q_norm"], s.q_mean) @ p["w_uq"].T
    q = q.reshape(T, H, s.head_dim + R)
    c = normed(down[:, s.q_rank:s.q_rank + K], p["kv_norm"], s.kv_mean)
    turns = p["turns"]

    def turned(x, t):
        out = x.copy()
        angle = 2 * np.pi * (first + t) * turns[:R // 2]
        out[..., 0::2] = x[..., 0::2] * np.cos(angle) - x[..., 1::2] * np.sin(angle)
        out[..., 1::2] = x[..., 1::2] * np.cos(angle) + x[..., 0::2] * np.sin(angle)
        return out

    row = np.concatenate([c, np.stack([turned(down[t, s.q_rank + K:], t)
                                       for t in range(T)])], axis=1)
    uk_t = p["w_uk_t"].reshape(H, K, s.head_dim)
    uv = p["w_ukv"].reshape(H, s.head_dim + s.head_vdim, K)[:, s.head_dim:]
    out = np.zeros((T, H, s.head_vdim))
    for t in range(T):
        low = max(0, t - s.window + 1)
        for a in range(H):
            query = np.concatenate([uk_t[a] @ q[t, a, :s.head_dim],
                                    turned(q[t, a, s.head_dim:], t)])
            e = row[low:t + 1] @ query * s.scale
            e = np.exp(e - e.max())
            out[t, a] = uv[a] @ (e / e.sum() @ c[low:t + 1])
    return out.reshape(T, -1)


def packed_linear(p, s, h):
    T, H, P, U = h.shape[0], s.heads, s.head_dim, s.head_vdim
    y = h @ p["w_in"].astype(np.float64).T
    part = lambda at, n: y[:, at:at + H * n].reshape(T, H, n)
    z = y[:, s.a1_row:] @ p["a2"].T + p["a2_bias"]
    alpha = plain.sigmoid(z).reshape(T, H, P) ** (1.0 / s.tau)
    o = np.stack([plain.recurrence(part(0, P)[:, a] * s.scale, part(s.k_row, P)[:, a],
                                   part(s.v_row, U)[:, a], alpha[:, a])[0]
                  for a in range(H)], axis=1)
    o = o / np.sqrt((o * o).sum(2, keepdims=True) / s.vdim + 1e-4) * p["o_norm"]
    g = part(s.gate_row, U)
    return (o * g * plain.sigmoid(g)).reshape(T, -1)


@pytest.mark.parametrize("name", sorted(models_of.CONFIGS))
def test_packed_arrays_multiply_out_to_the_layer(name):
    cfg = copy.deepcopy(models_of.CONFIGS[name])
    cfg["norm"]["eps"] = 1e-4
    w = models_of.weights(cfg, seed=3)
    parsed = vamalix.VamalixConfig.from_dict(cfg)
    assert parsed.dim % 64 == 0 and parsed.vocab_rows % 8 == 0
    W, S = cfg["width"], cfg["streams"]
    x = rng.standard_normal((S, 9, W))
    for i, s in enumerate(parsed.layers):
        if s.kind != MIXER_LATENT:
            s.set_rank(w["l%d.mix.a1" % i].shape[0])
        p = vamalix.pack_layer(s, W, parsed.dim, S,
                               lambda n, sh: models_of.getter(w)("l%d.%s" % (i, n), sh))
        assert p["w_in"].shape == (s.in_rows, parsed.dim) and s.in_rows % 8 == 0
        assert p["w_o"].shape == (parsed.dim, s.out_cols) and s.out_cols % 64 == 0

        def sublayer(full, q, f):
            h_in, mix, out = (a.astype(np.float64) for a in p["hc%d" % q])
            u = np.tensordot(h_in, full, 1)
            h = u / np.sqrt((u * u).sum(1, keepdims=True) / W + 1e-4) * p["norm%d" % q]
            return plain.mixed_streams(full, f(h), mix, out)

        full = np.zeros((S, 9, parsed.dim))
        full[:, :, :W] = x
        mixer = (lambda h: packed_latent(p, s, h, 4)) if s.kind == MIXER_LATENT else \
            (lambda h: packed_linear(p, s, h))
        full = sublayer(full, 1, lambda h: mixer(h) @ p["w_o"].T)
        if s.ff:
            assert s.hidden % 64 == 0
            full = sublayer(full, 2, lambda h: plain.gelu(h @ p["w_up"].T) @ p["w_down"].T)
        want = plain.layer(x, 4, w, cfg, i)
        assert np.abs(full[:, :, :W] - want).max() < 1e-5 * np.abs(want).max()
        assert not full[:, :, W:].any()


def test_what_a_configuration_may_not_say():
    def broken(change):
        cfg = copy.deepcopy(models_of.UNEVEN)
        change(cfg)
        with pytest.raises(ValueError):
            vamalix.VamalixConfig.from_dict(cfg)
    broken(lambda c: c.update(architecture="other"))
    broken(lambda c: c["layers"][0].update(type="recurrent"))
    broken(lambda c: c["layers"][0]["mixer"]["rot"].update(dims=4))
    broken(lambda c: c["layers"][0]["mlp"].update(kind="experts"))
    broken(lambda c: c.update(loop={"start": 2, "stop": 9, "times": 2}))
    broken(lambda c: c.update(loop={"start": 3, "stop": 2, "times": 2}))


def test_rank_of_the_decays_is_what_the_file_holds(tmp_path):
    cfg = models_of.ODD
    w = models_of.weights(cfg)
    models_of.write(str(tmp_path), cfg, w)
    text = (tmp_path / "config.json").read_text()
    assert '"_rank"' not in text and json.loads(text)["architecture"] == "Vamalix"
    f = safetensors.SafeTensors(str(tmp_path / "model.safetensors"))
    assert f.shape("l1.mix.a1") == (3, 77)
    with pytest.raises(ValueError):
        f.shape("absent")
    assert models.architecture_of(str(tmp_path)) == "Vamalix"
    assert models.library(str(tmp_path)).endswith(".so")


def test_the_configuration_struct_holds_a_layer_as_often_as_it_runs(monkeypatch):
    """What the library is handed, without the library."""
    cfg = vamalix.VamalixConfig.from_dict(models_of.UNEVEN)
    for i, s in enumerate(cfg.layers):
        if s.kind != MIXER_LATENT:
            s.set_rank(models_of.UNEVEN["layers"][i]["_rank"])
    seen = {}
    monkeypatch.setattr(vamalix.Decoder, "from_config",
                        classmethod(lambda cls, c, keep=None: seen.update(c=c, keep=keep)))
    layers = {i: dict(w_in=1000 + i, hc1=(1, 2, 3)) for i in range(4)}
    vamalix.decoder_of(cfg, dict(layers=layers, embed=1, head=2, final_norm=3), True, 50)
    c = seen["c"]
    assert c.n_layers == 6 and c.streams == 3 and c.dim == 128 and c.vocab_rows == 160
    assert [c.layers[i].w_in for i in range(6)] == [1000, 1001, 1002, 1001, 1002, 1003]
    assert (c.layers[0].q_rank, c.layers[0].q_mean, c.layers[0].kv_mean) == (64, 50, 70)
    assert (c.layers[0].hc1.hc_in, c.layers[0].hc1.mix, c.layers[0].hc1.out) == (1, 2, 3)
    assert c.layers[1].a_rank == 8 and c.layers[1].v_mean == 20
    assert abs(c.layers[1].scale - 12 ** -0.5) < 1e-7
