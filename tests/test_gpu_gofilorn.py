"""Gofilorn on the GPU against the plain restatement (oracle/gofilorn.py), through
the decoder's own entry points: portions of prompts, steps, rings that wrap,
window edges, shared tensors, batches, greedy generation and the trace runner."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import gofilorn as plain
from tests import gofilorn_models as models_of

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOLERANCE = 1e-5   # of the logits' root mean square: f32 sums in another order
DTYPES = ["bfloat16", "float32"]


def decoder(cfg, w, dtype="bfloat16", max_seq=320, batch=1, prefill_rows=0):
    from vx_b200 import gofilorn
    return gofilorn.from_tensors(gofilorn.GofilornConfig.from_dict(cfg),
                                 models_of.getter(w), dtype, max_seq, batch,
                                 prefill_rows)


def tokens_for(cfg, n, seed=2):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def close(got, want):
    assert got.shape == want.shape
    scale = np.sqrt(np.mean(want ** 2))
    err = np.sqrt(np.mean((got - want) ** 2, axis=1)) / scale
    assert np.isfinite(err).all() and err.max() < TOLERANCE, (err.argmax(), err.max())


def cut(n, sizes):
    """0..n in portions of the sizes, over and over."""
    at, i, out = 0, 0, []
    while at < n:
        out.append((at, min(n, at + sizes[i % len(sizes)])))
        at, i = out[-1][1], i + 1
    return out


def feed_all(d, tokens, portions):
    rows = [d.feed(tokens[a:b], range(b - a)) for a, b in portions]
    return np.concatenate(rows)


def status_ok():
    from vx_b200 import ops
    assert ops.kernel_status() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(models_of.CONFIGS))
def test_prompts_steps_and_portions(name, dtype):
    """The same tokens as one prompt, token by token, and in portions of several
    sizes down to two, on one decoder whose cache is used again each time."""
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


def test_a_request_after_a_longer_one_sees_nothing_of_it():
    cfg = models_of.EVEN
    w = models_of.weights(cfg, seed=4)
    d = decoder(cfg, w, prefill_rows=32)
    d.feed(tokens_for(cfg, 290, seed=9))
    d.reset()
    tokens = tokens_for(cfg, 40, seed=10)
    close(feed_all(d, tokens, cut(40, [7, 1, 1])), plain.logits(tokens, w, cfg))
    d.close()


@pytest.mark.parametrize("window", [1, 2, 16, 63, 64, 65, 100])
def test_keys_at_the_edge_of_the_window(window):
    """One key that takes most of the weight of every query that sees it, asked for
    from the last position that does and from the first that does not: in a prompt,
    in portions that begin or end there, and in steps."""
    for kv_heads in (1, 2):
        cfg, w, token = models_of.marked(window, kv_heads=kv_heads)
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


def test_mechanisms_one_by_one():
    """Models in which a single part is left: the embedding with its position and
    norm; attention with its gate; the feed-forward; a gain; the gate alone."""
    base = models_of.config(72, 90, [models_of.layer(3, 1, 24, 12, 0.5, 40)],
                            eps=0.02, embed_scale=0.7)
    tokens = tokens_for(base, 60)
    for zero, extra in ((("mix.o", "mlp.down"), {}), (("mlp.down",), {}),
                        (("mix.o",), {}), (("mix.q", "mlp.down"), {}),
                        (("mix.g", "mlp.down"), {}), (("mix.k",), {})):
        w = models_of.weights(base, seed=21, norm=0.8)
        for name in zero:
            w["l0." + name] = np.zeros_like(w["l0." + name])
        want = plain.logits(tokens, w, base)
        for dtype in DTYPES:
            d = decoder(base, w, dtype)
            close(feed_all(d, tokens, [(0, 60)]), want)
            d.reset()
            close(feed_all(d, tokens, cut(60, [1])), want)
            d.close()


def test_positions_far_along():
    """The sinusoid of the position at thousands, in a prompt and in steps; a ring
    far shorter than the sequence."""
    cfg = models_of.config(64, 50, [models_of.layer(2, 1, 16, 6, 0.3, 32)])
    w = models_of.weights(cfg)
    n = 9000
    tokens = tokens_for(cfg, n)
    d = decoder(cfg, w, max_seq=n + 8, prefill_rows=512)
    d.feed(tokens[:n - 40])
    got = np.concatenate([d.feed(tokens[n - 40:n - 20], range(20)),
                          feed_all(d, tokens[n - 20:], cut(20, [1]))])
    first = n - 60                 # a window of 6 does not reach further back
    x = plain.embed(tokens[first:], first, w["embed"], cfg["embedding"]["scale"],
                    w["embed.norm"], cfg["norm"]["eps"])
    x = plain.layer(x, w, cfg, 0)
    want = plain.rms_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T
    close(got, want[20:])
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
    """A step of several sequences gives each what it gets alone; the widths are
    such that sixteen rows do and do not fit the fused norm."""
    for cfg in (models_of.UNEVEN,
                models_of.config(1600, 72, [models_of.layer(4, 2, 24, 9, 0.3, 96)])):
        w = models_of.weights(cfg, seed=5)
        n = 26 if cfg is models_of.UNEVEN else 12
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
    """More wanted places than go through the classifier together, and few of many."""
    cfg = models_of.config(64, 37, [models_of.layer(2, 1, 16, 10, 0.3, 32)])
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
    want = plain.greedy(prompt, 40, w, cfg)
    d = decoder(cfg, w, dtype, prefill_rows=16)
    assert d.generate(prompt, 40) == want
    d.reset()
    assert d.generate(prompt[:1], 12) == plain.greedy(prompt[:1], 12, w, cfg)
    d.close()


def test_rings_handed_from_one_decoder_to_another():
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
    from vx_b200 import gofilorn
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
    big = models_of.config(64, 40, [models_of.layer(1, 1, 520, 4, 0.1, 0)])
    with pytest.raises(ValueError):
        decoder(big, models_of.weights(big))
    assert gofilorn.DTYPES == ("bfloat16", "float32")


def test_token_outside_the_table_gives_nan_and_leaves_no_trace():
    cfg = models_of.UNEVEN
    w = models_of.weights(cfg)
    d = decoder(cfg, w)
    bad = tokens_for(cfg, 30)
    bad[4] = cfg["vocab"]          # the first row of filling
    assert np.isnan(d.feed(bad, [4, 29])[0]).all()
    d.feed([cfg["vocab"] + 3])
    d.reset()
    tokens = tokens_for(cfg, 30)
    close(feed_all(d, tokens, [(0, 20)] + cut(30, [1])[20:]), plain.logits(tokens, w, cfg))
    d.close()


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
