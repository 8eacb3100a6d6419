"""Small Vamalix models for the tests: configurations, weights that are bf16 values,
and a safetensors file of them."""
import json
import math
import os

import numpy as np

from tests.gofilorn_models import bf16, getter, write as write_tensors


def latent(heads, dim, rot, vdim, q_rank, kv_rank, window, scale, ff=0, base=10000.0):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim,
                      "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot}, "mask": {"size": window}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def linear(heads, dim, vdim, tau, rank, ff=0):
    """`rank` is no entry of a config.json: only the tensors' shapes tell it."""
    return {"type": "gla", "_rank": rank,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, streams=2, loop=None, eps=1e-5, embed_scale=1.0,
           logit_scale=1.0, cap=20.0):
    return {"architecture": "Vamalix", "width": width, "vocab": vocab,
            "streams": streams, "loop": loop, "embedding": {"scale": embed_scale},
            "norm": {"eps": eps}, "logit_scale": logit_scale, "logit_softcap": cap,
            "layers": layers}


def shapes(cfg):
    W, S, out = cfg["width"], cfg["streams"], {}
    out["embed"] = out["head"] = (cfg["vocab"], W)
    out["final.norm"] = (W,)
    for i, entry in enumerate(cfg["layers"]):
        m, n = entry["mixer"], "l%d." % i
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if entry["type"] == "latent_attention":
            R, Q, K = m["rot_dim"], m["q_rank"], m["kv_rank"]
            out.update({n + "mix.dq": (Q, W), n + "mix.dq.norm": (Q,),
                        n + "mix.uq": (H * (D + R), Q), n + "mix.dkv": (K + R, W),
                        n + "mix.dkv.norm": (K,), n + "mix.uk": (H * D, K),
                        n + "mix.uv": (H * V, K)})
        else:
            A = entry["_rank"]
            out.update({n + "mix.q": (H * D, W), n + "mix.k": (H * D, W),
                        n + "mix.v": (H * V, W), n + "mix.g": (H * V, W),
                        n + "mix.a1": (A, W), n + "mix.a2": (H * D, A),
                        n + "mix.a2.b": (H * D,), n + "mix.norm": (V,)})
        out[n + "mix.o"] = (W, H * V)
        if entry["mlp"]:
            out[n + "mlp.up"] = (entry["mlp"]["ff"], W)
            out[n + "mlp.down"] = (W, entry["mlp"]["ff"])
        for q in (1, 2) if entry["mlp"] else (1,):
            out[n + "norm%d" % q] = (W,)
            out.update({n + "hc%d.in" % q: (S,), n + "hc%d.out" % q: (S,),
                        n + "hc%d.mix" % q: (S, S)})
    return out


def weights(cfg, seed=1, gain=1.2):
    """Matrices that keep the size of what they are applied to, gains around 1, decays
    of all sizes, and streams that differ and are far from symmetric in mixing."""
    rng = np.random.default_rng(seed)
    S, out = cfg["streams"], {}
    for name, shape in shapes(cfg).items():
        w = rng.standard_normal(shape)
        part = name.split(".", 1)[-1]
        if part == "mix.a2.b":
            w = 2.0 * w
        elif part.endswith("norm") or part in ("norm1", "norm2"):
            w = 1.0 + 0.3 * w
        elif part.endswith(".in"):
            w = (1.0 + 0.4 * w) / S
        elif part.endswith(".out"):
            w = 1.0 + 0.3 * w
        elif part.startswith("hc"):
            w = 0.85 * np.eye(S) + 0.3 * w / S
        elif part in ("mix.a1", "mix.a2"):
            w = 1.5 * w / math.sqrt(shape[1])
        elif name != "embed":
            w = gain * w / math.sqrt(shape[1])
        out[name] = bf16(w)
    return out


def shape_of(w):
    return lambda name: w[name].shape


def write(folder, cfg, w):
    write_tensors(folder, cfg, w)
    plain = dict(cfg, layers=[{k: v for k, v in entry.items() if k != "_rank"}
                              for entry in cfg["layers"]])
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(plain, f)


# sizes that are no multiple of anything the kernels work in, layers that differ in
# everything, feed-forwards after either mixer or none, a loop over both kinds
UNEVEN = config(84, 157, [
    latent(3, 20, 6, 28, 50, 70, 7, 0.25, ff=50, base=500.0),
    linear(5, 12, 20, 3.0, 5),
    latent(4, 10, 14, 9, 33, 41, 19, 0.3),
    linear(3, 36, 24, 16.0, 12, ff=70),
], streams=3, loop={"start": 1, "stop": 3, "times": 2}, eps=3e-3, embed_scale=1.7,
    logit_scale=2.5, cap=9.0)
# (An eps that is not tiny where a head's output can cancel to almost nothing: the norm
# behind it would blow up the rounding of the restatement and of the kernels alike.)
# one stream, no loop, one head, one layer of a kind
SMALL = config(40, 33, [
    linear(1, 8, 16, 1.0, 1, ff=24),
    latent(1, 4, 2, 8, 12, 10, 3, 0.6, ff=16),
], streams=1)
EVEN = config(128, 320, [
    latent(8, 64, 32, 64, 128, 192, 33, 0.1, ff=192),
    linear(4, 64, 128, 8.0, 16),
    latent(16, 32, 32, 32, 64, 64, 50, 0.12, ff=256, base=1e6),
], streams=4, loop={"start": 0, "stop": 3, "times": 2}, eps=1e-2)
# heads, latents and states of the larger forms of the kernels; eight and nine streams
WIDE = config(192, 96, [
    latent(2, 136, 40, 120, 200, 300, 40, 0.08, ff=64),
    linear(2, 200, 264, 5.0, 20),
    latent(1, 264, 64, 200, 96, 448, 25, 0.06),
    latent(5, 24, 72, 300, 100, 700, 90, 0.1),
], streams=8)
WIDER = config(72, 51, [
    linear(1, 400, 40, 12.0, 24),
    latent(2, 300, 100, 400, 40, 520, 12, 0.05),
    linear(3, 100, 600, 2.0, 9),
], streams=9)
ODD = config(77, 101, [latent(7, 9, 10, 5, 21, 23, 90, 0.3, ff=21),
                       linear(7, 3, 5, 4.0, 3, ff=65)], streams=5)
CONFIGS = {"uneven": UNEVEN, "small": SMALL, "even": EVEN, "wide": WIDE,
           "wider": WIDER, "odd": ODD}


def marked(window, heads=4, layers=1, ff=40, streams=2, width=96, vocab=61):
    """A model of latent attention and a token such that every query scores that
    token's key far above any other: where the token is seen at all, it takes most of
    the weight. Returns (config, weights, the token)."""
    dim, rot, rank = 32, 8, 48
    cfg = config(width, vocab, [latent(heads, dim, rot, 24, rank, rank, window, 0.3,
                                       ff=ff)] * layers, streams=streams, embed_scale=3.0)
    w = weights(cfg, seed=11)
    rng = np.random.default_rng(12)
    token = vocab - 1
    # all other tokens share a direction, which the queries are made from
    common = rng.standard_normal(width)
    mark = rng.standard_normal(width)
    mark -= mark @ common / (common @ common) * common
    table = 0.4 * rng.standard_normal((vocab, width)) + common
    table[token] = 1.2 * mark
    w["embed"] = bf16(table)
    unit = lambda v: v / np.sqrt((v * v).mean())
    for i in range(layers):
        n = "l%d." % i
        for q in ("norm1", "mix.dq.norm", "mix.dkv.norm"):
            w[n + q] = np.ones_like(w[n + q])
        # the marked token's latent, and queries along the key each head makes of it
        latent_of_mark = unit(w[n + "mix.dkv"][:rank] @ unit(mark))
        q_of_common = unit(w[n + "mix.dq"] @ unit(common))
        uq = np.zeros((heads, dim + rot, rank))
        for h in range(heads):
            key = w[n + "mix.uk"][h * dim:(h + 1) * dim] @ latent_of_mark
            uq[h, :dim] = 8.0 * np.outer(unit(key), q_of_common) / rank
        w[n + "mix.uq"] = bf16(uq.reshape(-1, rank))
    return cfg, w, token


def slow_decays(bias=6.0, eps=1e-5):
    """Layers of gated linear attention that forget so slowly that the first tokens are
    still read hundreds of tokens on."""
    cfg = config(64, 47, [linear(2, 16, 24, 8.0, 4), linear(3, 40, 16, 8.0, 6, ff=48)],
                 loop={"start": 0, "stop": 1, "times": 2}, eps=eps)
    w = weights(cfg, seed=31)
    for i in range(2):
        w["l%d.mix.a2.b" % i] = np.full_like(w["l%d.mix.a2.b" % i], bias)
        w["l%d.mix.a2" % i] = bf16(0.2 * w["l%d.mix.a2" % i])
    return cfg, w
