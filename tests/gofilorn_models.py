"""Small Gofilorn models for the tests: configurations, weights that are bf16
values, and a safetensors file of them."""
import json
import os
import struct

import numpy as np


def layer(heads, kv_heads, dim, window, scale, ff, weights_of=None):
    entry = {"type": "attention",
             "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim,
                       "mask": {"size": window}, "scale": scale},
             "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def config(width, vocab, layers, eps=1e-5, embed_scale=2.0):
    return {"architecture": "Gofilorn", "width": width, "vocab": vocab,
            "embedding": {"scale": embed_scale}, "norm": {"eps": eps},
            "layers": layers}


def bf16(a):
    """The nearest bf16 values, as f64."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.view(np.float32).astype(np.float64)


def shapes(cfg):
    width, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], width)
    out["embed.norm"] = out["final.norm"] = (width,)
    for i, entry in enumerate(cfg["layers"]):
        if "weights_of" in entry:
            continue
        m, n = entry["mixer"], "l%d." % i
        out[n + "norm1"] = (width,)
        out[n + "mix.q"] = out[n + "mix.g"] = (m["heads"] * m["dim"], width)
        out[n + "mix.k"] = (m["kv_heads"] * m["dim"], width)
        out[n + "mix.o"] = (width, m["heads"] * m["dim"])
        if entry["mlp"]:
            out[n + "mlp.up"] = (entry["mlp"]["ff"], width)
            out[n + "mlp.down"] = (width, entry["mlp"]["ff"])
    return out


def weights(cfg, seed=1, gain=1.2, norm=0.3):
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        w = rng.standard_normal(shape)
        if len(shape) == 1:
            w = norm * w
        elif name != "embed":
            w = gain * w / np.sqrt(shape[1])
        out[name] = bf16(w)
    return out


def getter(w):
    """The tensor(name, shape) that the loader asks."""
    def get(name, shape):
        a = w[name]
        assert a.shape == tuple(shape), (name, a.shape, shape)
        return a.astype(np.float32)
    return get


def write(folder, cfg, w):
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {"__metadata__": {"format": "pt"}}, [], 0
    for name, a in w.items():
        b = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2")
        head[name] = {"dtype": "BF16", "shape": list(a.shape),
                      "data_offsets": [at, at + b.nbytes]}
        at += b.nbytes
        blobs.append(b.tobytes())
    text = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))


# sizes that are no multiple of anything the kernels work in, layers that differ,
# layers without a feed-forward, tensors used twice
UNEVEN = config(84, 157, [
    layer(4, 2, 20, 7, 0.4, 50),
    layer(3, 1, 36, 20, 0.21, 0),
    layer(6, 6, 12, 1, 1.0, 33),
    layer(4, 2, 20, 11, 0.3, 50, weights_of=0),
    layer(3, 1, 36, 20, 0.21, 0, weights_of=1),
], eps=3e-3, embed_scale=1.5)
EVEN = config(128, 320, [
    layer(10, 5, 32, 33, 0.18, 192),
    layer(4, 1, 128, 64, 0.09, 320),
    layer(10, 5, 32, 33, 0.18, 192, weights_of=0),
], embed_scale=1.0)
WIDE_HEADS = config(192, 96, [
    layer(2, 1, 136, 40, 0.1, 64),
    layer(5, 1, 264, 25, 0.07, 0),
    layer(1, 1, 256, 300, 0.06, 72),
])
ODD_WIDTH = config(77, 101, [layer(2, 2, 9, 5, 0.5, 21), layer(7, 1, 64, 90, 0.125, 65)])
CONFIGS = {"uneven": UNEVEN, "even": EVEN, "wide_heads": WIDE_HEADS,
           "odd_width": ODD_WIDTH}


def marked(window, kv_heads=1, heads=4, dim=32, width=96, vocab=61, layers=1, ff=40):
    """A model and a token such that every query scores that token's key far above
    any other: where the token is seen at all, it takes most of the weight. Returns
    (config, weights, the token)."""
    cfg = config(width, vocab, [layer(heads, kv_heads, dim, window, 0.35, ff)] * layers,
                 embed_scale=6.0)
    w = weights(cfg, seed=11, norm=0.0)
    rng = np.random.default_rng(12)
    common = rng.standard_normal(width)
    token = vocab - 1
    table = 0.5 * rng.standard_normal((vocab, width)) + common
    mark = rng.standard_normal(width)
    mark -= mark @ common / (common @ common) * common
    table[token] = 1.1 * mark
    w["embed"] = bf16(table)
    for i in range(layers):
        n = "l%d." % i
        keys = w[n + "mix.k"] @ (mark / np.sqrt((mark * mark).mean()))
        keys = keys.reshape(kv_heads, dim)
        q = np.zeros((heads, dim, width))
        for h in range(heads):
            k = keys[h // (heads // kv_heads)]
            q[h] = 9.0 * np.outer(k / np.linalg.norm(k),
                                  common / np.linalg.norm(common)) / np.sqrt(width)
        w[n + "mix.q"] = bf16(q.reshape(heads * dim, width))
    return cfg, w, token
