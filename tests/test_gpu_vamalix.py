"""Vamalix on the GPU against the plain restatement (oracle/vamalix.py), through the
decoder's own entry points: portions of prompts, steps, rings that wrap, window edges,
states that are carried and given back, loops, batches, greedy generation and the trace
runner; and each mechanism's kernel alone."""
import copy
import ctypes as C
import json
import os
import subprocess

import numpy as np
import pytest

from oracle import vamalix as plain
from tests import vamalix_models as models_of
from tests.test_gpu_gofilorn import cut, feed_all, status_ok, tokens_for

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# of the logits' root mean square: f32 sums in another order, through a dozen
# sublayers that each divide by a norm
TOLERANCE = 3e-5
DTYPES = ["bfloat16", "float32"]


def decoder(cfg, w, dtype="bfloat16", max_seq=320, batch=1, prefill_rows=0):
    from vx_b200 import vamalix
    return vamalix.from_tensors(vamalix.VamalixConfig.from_dict(cfg),
                                models_of.getter(w), models_of.shape_of(w), dtype,
                                max_seq, batch, prefill_rows)


def close(got, want, tolerance=TOLERANCE):
    assert got.shape == want.shape
    scale = np.sqrt(np.mean(want ** 2))
    err = np.sqrt(np.mean((got - want) ** 2, axis=1)) / scale
    assert np.isfinite(err).all() and err.max() < tolerance, (err.argmax(), err.max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(models_of.CONFIGS))
def test_prompts_steps_and_portions(name, dtype):
    """The same tokens as one prompt, token by token, and in portions of several
    sizes down to two, on one decoder whose rings and states are used again."""
    cfg = models_of.CONFIGS[name]
    w = models_of.weights(cfg)
    tokens = tokens_for(cfg, 150)
    want = plain.logits(tokens, w, cfg)
    d = decoder(cfg, w, dtype)
    for sizes in ([150], [1], [2], [3, 1, 2, 40], [33, 64, 5], [149, 1]):
        d.reset()
        close(feed_all(d, tokens, cut(len(tokens), sizes)), want)
    d.close()
    status_ok()


@pytest.mark.parametrize("dtype", DTYPES)
def test_rings_that_wrap(dtype):
    """Rings of a window and sixteen rows: longer portions go through in pieces,
    and every ring is overwritten many times."""
    cfg = models_of.UNEVEN
    w = models_of.weights(cfg, seed=8)
    tokens = tokens_for(cfg, 310)
    want = plain.logits(tokens, w, cfg)
    d = decoder(cfg, w, dtype, max_seq=310, prefill_rows=16)
    for sizes in ([310], [16], [17, 1, 5], [1], [61, 1, 1, 1]):
        d.reset()
        close(feed_all(d, tokens, cut(len(tokens), sizes)), want)
    d.close()


@pytest.mark.parametrize("name", ["even", "small"])
def test_a_request_after_a_longer_one_sees_nothing_of_it(name):
    cfg = models_of.CONFIGS[name]
    w = models_of.weights(cfg, seed=4)
    d = decoder(cfg, w, prefill_rows=32)
    d.feed(tokens_for(cfg, 290, seed=9))
    tokens = tokens_for(cfg, 40, seed=10)
    want = plain.logits(tokens, w, cfg)
    for sizes in ([7, 1, 1], [1], [40]):
        d.reset()
        close(feed_all(d, tokens, cut(40, sizes)), want)
    d.close()


@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 100])
def test_keys_at_the_edge_of_the_window(window):
    """One key that takes most of the weight of every query that sees it, asked for
    from the last position that does and from the first that does not: in a prompt,
    in portions that begin or end there, and in steps."""
    for heads in (1, 5):
        cfg, w, token = models_of.marked(window, heads=heads)
        n = window + 40
        tokens = np.random.default_rng(3).integers(0, cfg["vocab"] - 1, n)
        tokens[9] = token
        want = plain.logits(tokens, w, cfg)
        edge = 9 + window          # the first position that does not see it
        d = decoder(cfg, w, prefill_rows=24)
        wide = decoder(cfg, w)
        for portions in ([(0, n)], cut(n, [1]), [(0, edge), (edge, n)],
                         [(0, edge - 1)] * (edge > 1) + [(edge - 1, edge + 1),
                                                         (edge + 1, n)]):
            for which in (d, wide):
                which.reset()
                close(feed_all(which, tokens, portions), want)
        d.close()
        wide.close()


def test_a_key_far_back_in_a_long_window():
    cfg, w, token = models_of.marked(250, layers=2)
    tokens = np.random.default_rng(6).integers(0, cfg["vocab"] - 1, 300)
    tokens[30] = token
    want = plain.logits(tokens, w, cfg)
    for dtype in DTYPES:
        d = decoder(cfg, w, dtype)
        close(feed_all(d, tokens, [(0, 300)]), want)
        d.reset()
        close(feed_all(d, tokens, [(0, 64), (64, 128), (128, 270)]
                       + cut(300, [1])[270:]), want)
        d.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_states_that_forget_slowly(dtype):
    """The first tokens still read hundreds of tokens on, through portions and steps."""
    cfg, w = models_of.slow_decays()
    tokens = tokens_for(cfg, 300)
    want = plain.logits(tokens, w, cfg)
    d = decoder(cfg, w, dtype)
    for sizes in ([300], [1], [2, 1, 37], [100, 15, 17], [16, 8, 9]):
        d.reset()
        close(feed_all(d, tokens, cut(300, sizes)), want)
    d.close()


def test_states_that_forget_at_once():
    """Decays as small as f32 holds, and exactly zero, for z far below zero."""
    cfg, w = models_of.slow_decays(bias=-60.0, eps=1e-2)
    cfg = copy.deepcopy(cfg)
    cfg["layers"][1]["mixer"]["tau"] = 0.5
    tokens = tokens_for(cfg, 60)
    want = plain.logits(tokens, w, cfg)
    d = decoder(cfg, w)
    for sizes in ([60], [1], [5, 1]):
        d.reset()
        close(feed_all(d, tokens, cut(60, sizes)), want)
    d.close()


def test_mechanisms_one_by_one():
    """Models in which a single part is left: a mixer, a feed-forward, the rotated or
    the unrotated part of the scores, the gate, the mixing alone."""
    both = models_of.config(72, 90, [
        models_of.latent(3, 24, 8, 16, 40, 48, 12, 0.5, ff=40, base=50.0),
        models_of.linear(2, 24, 40, 4.0, 6, ff=56)], streams=3, eps=0.02,
        embed_scale=0.7, logit_scale=3.0, cap=4.0)
    tokens = tokens_for(both, 60)
    base = models_of.weights(both, seed=21)
    H = 3

    def rows_of(name, keep):
        def change(w):
            a = w[name].reshape(H, -1, w[name].shape[1]).copy()
            a[:, slice(24) if keep == "rotated" else slice(24, None)] = 0
            w[name] = a.reshape(w[name].shape)
        return change

    def zero(*names):
        def change(w):
            for n in names:
                w[n] = np.zeros_like(w[n])
        return change

    for change in (zero("l0.mix.o", "l1.mix.o"), zero("l0.mlp.down", "l1.mlp.down"),
                   zero("l0.mix.o", "l0.mlp.down", "l1.mlp.down"),
                   zero("l1.mix.o", "l0.mlp.down", "l1.mlp.down"),
                   zero("l0.mix.o", "l0.mlp.down", "l1.mix.o", "l1.mlp.down"),
                   zero("l0.mix.uq"), zero("l1.mix.a1"), zero("l1.mix.a2.b"),
                   rows_of("l0.mix.uq", "rotated"), rows_of("l0.mix.uq", "unrotated")):
        w = dict(base)
        change(w)
        want = plain.logits(tokens, w, both)
        for dtype in DTYPES:
            d = decoder(both, w, dtype)
            close(feed_all(d, tokens, [(0, 60)]), want)
            d.reset()
            close(feed_all(d, tokens, cut(60, [1])), want)
            d.close()


@pytest.mark.parametrize("streams", [1, 2, 3, 4, 6, 8, 17, 32])
def test_any_number_of_streams(streams):
    cfg = copy.deepcopy(models_of.UNEVEN)
    cfg["streams"] = streams
    w = models_of.weights(cfg, seed=40 + streams)
    tokens = tokens_for(cfg, 40)
    want = plain.logits(tokens, w, cfg)
    d = decoder(cfg, w)
    for sizes in ([40], [1], [9, 1, 2]):
        d.reset()
        close(feed_all(d, tokens, cut(40, sizes)), want)
    d.close()


def test_positions_far_along():
    """Angles at thousands, in a prompt and in steps; a ring far shorter than the
    sequence. Only layers that forget: what lies further back than a window does not
    reach the end."""
    cfg = models_of.config(64, 50, [
        models_of.latent(2, 16, 16, 16, 32, 40, 6, 0.3, ff=32, base=30.0)])
    w = models_of.weights(cfg)
    n = 9000
    tokens = tokens_for(cfg, n)
    d = decoder(cfg, w, max_seq=n + 8, prefill_rows=512)
    d.feed(tokens[:n - 40])
    got = np.concatenate([d.feed(tokens[n - 40:n - 20], range(20)),
                          feed_all(d, tokens[n - 20:], cut(20, [1]))])
    first = n - 60
    want = plain.logits(tokens[first:], w, cfg, first)
    close(got, want[20:])
    assert np.abs(plain.logits(tokens[first:], w, cfg, first + 1) - want).max() < 1e-9
    d.close()


def test_long_decoding():
    cfg = models_of.UNEVEN
    w = models_of.weights(cfg, seed=13)
    tokens = tokens_for(cfg, 400)
    d = decoder(cfg, w, max_seq=400, prefill_rows=8)
    close(feed_all(d, tokens, [(0, 5)] + cut(400, [1])[5:]), plain.logits(tokens, w, cfg))
    d.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("batch", [2, 8, 16])
def test_sequences_side_by_side(batch, dtype):
    """A step of several sequences gives each what it gets alone; the widths are such
    that sixteen rows do and do not fit the norm in front of a projection."""
    wide = models_of.config(1600, 72, [
        models_of.latent(3, 24, 8, 16, 1600, 48, 9, 0.3, ff=96),
        models_of.linear(4, 24, 16, 4.0, 6)])
    for cfg in (models_of.UNEVEN, wide):
        w = models_of.weights(cfg, seed=5)
        n = 26 if cfg is models_of.UNEVEN else 10
        tokens = np.stack([tokens_for(cfg, n, seed=50 + b) for b in range(batch)])
        d = decoder(cfg, w, dtype, batch=batch)
        got = []
        for t in range(n):
            d.step(tokens[:, t])
            got.append(d.logits())
        got = np.stack(got, axis=1)
        for b in range(batch):
            close(got[b], plain.logits(tokens[b], w, cfg))
        d.close()


def test_wanted_places_of_a_long_portion():
    """More wanted places than go through the classifier together, few of many, and
    portions in which nothing is wanted and the last layer stops at its cache."""
    for last in (models_of.latent(2, 16, 8, 16, 32, 24, 10, 0.3, ff=32),
                 models_of.linear(2, 16, 24, 4.0, 6, ff=32)):
        cfg = models_of.config(64, 37, [models_of.linear(2, 8, 16, 9.0, 4), last])
        w = models_of.weights(cfg)
        tokens = tokens_for(cfg, 600)
        want = plain.logits(tokens, w, cfg)
        d = decoder(cfg, w, max_seq=600, prefill_rows=400)
        close(d.feed(tokens, range(600)), want)
        d.reset()
        places = [0, 1, 63, 64, 399, 400, 598, 599]
        close(d.feed(tokens, places), want[places])
        d.reset()
        assert d.feed(tokens[:50]).shape == (0, 37)
        close(d.feed(tokens[50:], [0, 549]), want[[50, 599]])
        d.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation(dtype):
    cfg = models_of.EVEN
    w = models_of.weights(cfg, seed=17)
    prompt = tokens_for(cfg, 37)
    want = plain.greedy(prompt, 30, w, cfg)
    d = decoder(cfg, w, dtype, prefill_rows=16)
    assert d.generate(prompt, 30) == want
    d.reset()
    assert d.generate(prompt[:1], 12) == plain.greedy(prompt[:1], 12, w, cfg)
    d.close()


def test_rings_and_states_handed_from_one_decoder_to_another():
    cfg = models_of.EVEN
    w = models_of.weights(cfg, seed=19)
    tokens = tokens_for(cfg, 220)
    want = plain.logits(tokens, w, cfg)
    for n in (20, 200):            # before and after the rings are full
        first, second = decoder(cfg, w, prefill_rows=16), decoder(cfg, w, prefill_rows=16)
        first.feed(tokens[:n])
        assert first.kv_cache(1) is None and first.kv_cache_bytes == second.kv_cache_bytes
        assert second.adopt_kv(first.kv_cache(0), first.kv_cache(1), n) == n
        first.close()
        close(feed_all(second, tokens[n:n + 20], [(0, 6)] + cut(20, [1])[6:]),
              want[n:n + 20])
        second.close()


def test_refusals():
    cfg = models_of.EVEN
    w = models_of.weights(cfg)
    d = decoder(cfg, w, max_seq=20)
    with pytest.raises(ValueError):
        d.feed(tokens_for(cfg, 21))
    with pytest.raises(ValueError):
        d.feed(tokens_for(cfg, 5), [3, 2])
    d.close()
    with pytest.raises(ValueError):
        decoder(cfg, w, dtype="float16")
    with pytest.raises(ValueError):
        decoder(cfg, w, batch=3)
    for layer in (models_of.latent(1, 500, 16, 8, 16, 16, 4, 0.1),
                  models_of.latent(1, 16, 16, 520, 16, 16, 4, 0.1),
                  models_of.latent(1, 16, 72, 16, 16, 980, 4, 0.1),
                  models_of.linear(1, 520, 8, 1.0, 4)):
        big = models_of.config(64, 40, [layer])
        with pytest.raises(ValueError):
            decoder(big, models_of.weights(big))


def test_token_outside_the_table_gives_nan_and_leaves_no_trace():
    cfg = models_of.UNEVEN
    w = models_of.weights(cfg)
    d = decoder(cfg, w)
    bad = tokens_for(cfg, 30)
    bad[4] = cfg["vocab"]          # the first row of filling
    assert np.isnan(d.feed(bad, [4, 29])[0]).all()
    d.feed([cfg["vocab"] + 3])
    tokens = tokens_for(cfg, 30)
    want = plain.logits(tokens, w, cfg)
    for sizes in ([20, 1], [1]):
        d.reset()
        close(feed_all(d, tokens, cut(30, sizes)), want)
    d.close()


def test_sizes_like_a_real_models_agree_between_prompt_and_steps():
    """Layers of real width, several of each kind, a prompt of many tiles right after
    shorter ones: the prompt's logits against the steps', which share no kernel."""
    from vx_b200 import vamalix
    latent = models_of.latent(16, 128, 64, 128, 768, 512, 256, 192 ** -0.5, ff=2048)
    linear = models_of.linear(4, 128, 256, 16.0, 16)
    cfg = vamalix.VamalixConfig.from_dict(models_of.config(
        1024, 2000, [latent, linear] * 3, streams=4, cap=30.0))
    d = vamalix.synthetic(cfg, 1200)
    tokens = tokens_for(dict(vocab=2000), 1100)
    for n in (512, 512, 64, 1000):
        d.reset()
        d.feed(tokens[:n])
    d.reset()
    prompt = d.feed(tokens, list(range(1000, 1100)))
    d.reset()
    d.feed(tokens[:1000])
    steps = np.concatenate([d.feed([t], [0]) for t in tokens[1000:]])
    close(prompt, steps, 2e-4)
    d.close()
    status_ok()


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(tmp_path, dtype):
    cfg = models_of.UNEVEN
    w = models_of.weights(cfg, seed=23)
    models_of.write(str(tmp_path), cfg, w)
    a, b = tokens_for(cfg, 60, seed=1), tokens_for(cfg, 9, seed=2)
    steps, expect = [], {}

    def say(request, tokens, lo, hi, want, end):
        n = len(steps)
        steps.append(json.dumps({"step": n, "end": [request] * end, "entries": [
            {"id": request, "tokens": [int(t) for t in tokens[lo:hi]], "want": want}]}))
        if want:
            expect[n] = plain.logits(tokens[:hi], w, cfg)[[lo + p for p in want]]

    say("a", a, 0, 20, [], False)
    say("a", a, 20, 58, [37, 0, 5], False)
    say("a", a, 58, 59, [0], False)
    say("a", a, 59, 60, [0], True)
    say("b", b, 0, 2, [1], False)
    say("b", b, 2, 9, [0, 6], True)
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model",
                        str(tmp_path), "--dtype", dtype, "--out", str(tmp_path),
                        "--max-tokens", "60"], input="\n".join(steps) + "\n", text=True,
                       capture_output=True, timeout=300)
    assert r.returncode == 0, r.stderr
    done = [line for line in r.stdout.splitlines() if line.startswith("done ")]
    assert done == ["done %d" % n for n in range(len(steps))]
    for n in range(len(steps)):
        path = tmp_path / ("%d.f32" % n)
        assert path.exists() == (n in expect)
        if n in expect:
            close(np.fromfile(path, "<f4").reshape(-1, cfg["vocab"]), expect[n])
