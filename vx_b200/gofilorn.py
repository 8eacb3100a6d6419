"""Gofilorn decoders on the whole-token entry points (vx_decoder_create_parallel,
include/vx_b200.h): what its config.json says, its weights in the layout of the
kernels, and synthetic models of the same architecture.

A layer adds mixer(h) + ff(h) to the residual, h being one RMSNorm of it:
attention over a sliding window whose keys are the values too, with no rotation,
a sigmoid gate on its output; ff = down(relu(up h)^2), or nothing.  A layer may
use another layer's tensors, with a cache of its own.
"""
import json
import os

import numpy as np

from . import abi
from .lib import ParallelConfig, ParallelLayer, lib
from .llama import Decoder
from .safetensors import SafeTensors, to_bf16

ARCHITECTURE = "Gofilorn"
DTYPES = ("bfloat16", "float32")


def _up(n, step):
    return (n + step - 1) // step * step


class LayerShape:
    """One layer: its sizes, and how the kernels lay its matrices out: heads
    filled up to 8 values, the output matrix's columns to 64."""

    def __init__(self, heads, kv_heads, dim, window, scale, ff, source):
        self.heads, self.kv_heads, self.dim = heads, kv_heads, dim
        self.window, self.scale, self.ff, self.source = window, scale, ff, source
        self.head_dim = _up(dim, 8)
        self.att = heads * self.head_dim
        self.hidden = _up(self.att + ff, 64) - self.att
        self.in_rows = 2 * self.att + kv_heads * self.head_dim + self.hidden
        self.out_cols = self.att + self.hidden

    def same_tensors(self, other):
        return (self.heads, self.kv_heads, self.dim, self.ff) == (
            other.heads, other.kv_heads, other.dim, other.ff)


class GofilornConfig:
    """What config.json says; `layers` holds a LayerShape each, `source` being
    the layer whose tensors it uses."""

    def __init__(self, width, vocab, eps, embed_scale, layers):
        self.width, self.vocab, self.eps = width, vocab, eps
        self.embed_scale, self.layers = embed_scale, layers
        self.dim, self.vocab_rows = _up(width, 64), _up(vocab, 8)

    @classmethod
    def from_dict(cls, config):
        if config.get("architecture") != ARCHITECTURE:
            raise ValueError("not a %s configuration: %r"
                             % (ARCHITECTURE, config.get("architecture")))
        layers = []
        for i, entry in enumerate(config["layers"]):
            if entry.get("type") != "attention":
                raise ValueError("layer %d has the type %r" % (i, entry.get("type")))
            m, mlp = entry["mixer"], entry.get("mlp")
            if m.get("vdim", m["dim"]) != m["dim"]:
                raise ValueError("layer %d: keys serve as values, so vdim must be dim" % i)
            if m["heads"] % m["kv_heads"]:
                raise ValueError("layer %d: heads is no multiple of kv_heads" % i)
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError("layer %d has a feed-forward of the kind %r"
                                 % (i, mlp.get("kind")))
            source = entry.get("weights_of")
            if source is None:
                source = i
            elif not 0 <= source < len(config["layers"]) or source == i:
                raise ValueError("layer %d: weights_of is %r" % (i, source))
            layers.append(LayerShape(m["heads"], m["kv_heads"], m["dim"],
                                     m["mask"]["size"], m["scale"],
                                     mlp["ff"] if mlp is not None else 0, source))
        named = [layer.source for layer in layers]
        for i, layer in enumerate(layers):
            for _ in layers:        # to the layer that has tensors of its own
                layer.source = named[layer.source]
            if named[layer.source] != layer.source or \
                    not layer.same_tensors(layers[layer.source]):
                raise ValueError("layer %d cannot use the tensors of layer %d"
                                 % (i, named[i]))
        return cls(config["width"], config["vocab"], config["norm"]["eps"],
                   config["embedding"]["scale"], layers)

    @classmethod
    def from_file(cls, path):
        with open(path) as f:
            return cls.from_dict(json.load(f))


def turns_per_position(width):
    """The part of a full turn that the angle of values 2i and 2i + 1 advances
    per position: 10000^(-2i / width) / (2 pi)."""
    i = np.arange((width + 1) // 2, dtype=np.float64)
    return 10000.0 ** (-2.0 * i / width) / (2.0 * np.pi)


def pack_layer(shape, width, dim, tensor):
    """(input matrix, output matrix) of a layer as f32. tensor(name, shape) gives
    the layer's tensors. Rows q | k | gate | up; columns attention | up; zeros
    fill heads up to head_dim, `up` to `hidden`, the width to dim."""
    H, G, D, P = shape.heads, shape.kv_heads, shape.dim, shape.head_dim

    def head_rows(name, heads):
        out = np.zeros((heads, P, dim), np.float32)
        out[:, :D, :width] = tensor(name, (heads * D, width)).reshape(heads, D, width)
        return out.reshape(heads * P, dim)

    up = np.zeros((shape.hidden, dim), np.float32)
    w_out = np.zeros((dim, shape.out_cols), np.float32)
    w_out[:width, :shape.att].reshape(width, H, P)[:, :, :D] = \
        tensor("mix.o", (width, H * D)).reshape(width, H, D)
    if shape.ff:
        up[:shape.ff, :width] = tensor("mlp.up", (shape.ff, width))
        w_out[:width, shape.att:shape.att + shape.ff] = \
            tensor("mlp.down", (width, shape.ff))
    w_in = np.concatenate([head_rows("mix.q", H), head_rows("mix.k", G),
                           head_rows("mix.g", H), up])
    return w_in, w_out


def pack_gain(w, dim):
    """What multiplies the normalised value, 1 + w, in f32."""
    out = np.zeros(dim, np.float32)
    out[:w.shape[0]] = np.float32(1.0) + w.astype(np.float32)
    return out


def decoder_of(config, tensors, bf16, max_seq, batch=1, prefill_rows=0, keep=None):
    """A Decoder over device addresses: tensors["layers"] maps a layer that has
    tensors of its own to (norm, w_in, w_out); embed, embed_norm, final_norm and
    turns are addresses."""
    layers = (ParallelLayer * len(config.layers))()
    for to, s in zip(layers, config.layers):
        norm, w_in, w_out = tensors["layers"][s.source]
        to.q_heads, to.kv_heads, to.head_dim = s.heads, s.kv_heads, s.head_dim
        to.hidden, to.window, to.score_scale = s.hidden, s.window, s.scale
        to.norm, to.w_in, to.w_out = norm, w_in, w_out
    cfg = ParallelConfig(
        width=config.width, dim=config.dim, n_layers=len(config.layers),
        vocab=config.vocab, vocab_rows=config.vocab_rows, max_seq=max_seq,
        weights_bf16=1 if bf16 else 0, batch=batch, prefill_rows=prefill_rows,
        eps=config.eps, embed_scale=config.embed_scale, embed=tensors["embed"],
        classifier=tensors["embed"], embed_norm=tensors["embed_norm"],
        final_norm=tensors["final_norm"], turns=tensors["turns"], layers=layers)
    return Decoder.from_config(cfg, keep=(keep, layers))


def from_tensors(config, tensor, dtype="bfloat16", max_seq=4096, batch=1,
                 prefill_rows=0):
    """A Decoder of the weights that tensor(name, shape) gives as f32."""
    if dtype not in DTYPES:
        raise ValueError("the dtype is one of %s" % (DTYPES,))
    bf16 = dtype == "bfloat16"
    keep = []

    def place(a):
        t = abi.DeviceTensor.from_host(a)
        keep.append(t)
        return t.ptr

    def matrix(a):
        t = abi.DeviceTensor.from_host(to_bf16(a), bf16=True) if bf16 \
            else abi.DeviceTensor.from_host(a)
        keep.append(t)
        return t.ptr

    table = np.zeros((config.vocab_rows, config.dim), np.float32)
    table[:config.vocab, :config.width] = tensor("embed", (config.vocab, config.width))

    def gain(name):
        return place(pack_gain(tensor(name, (config.width,)), config.dim))

    owned = {}
    for i, shape in enumerate(config.layers):
        if shape.source != i:
            continue
        w_in, w_out = pack_layer(shape, config.width, config.dim,
                                 lambda name, sh: tensor("l%d.%s" % (i, name), sh))
        owned[i] = (gain("l%d.norm1" % i), matrix(w_in), matrix(w_out))
    tensors = dict(layers=owned, embed=matrix(table), embed_norm=gain("embed.norm"),
                   final_norm=gain("final.norm"),
                   turns=place(turns_per_position(config.width)))
    return decoder_of(config, tensors, bf16, max_seq, batch, prefill_rows, keep)


def load(path, dtype="bfloat16", max_seq=4096, batch=1, prefill_rows=0):
    """The model of a folder with config.json and model.safetensors."""
    config = GofilornConfig.from_file(os.path.join(path, "config.json"))
    weights = SafeTensors(os.path.join(path, "model.safetensors"))
    return from_tensors(config, weights.f32, dtype, max_seq, batch, prefill_rows)


def synthetic(config, max_seq, seed=7, batch=1, sigma=0.02, prefill_rows=0):
    """A bf16 model of random weights made on the GPU (torch only holds the
    memory): N(0, sigma^2) matrices, gains of 1. For measurements: where head,
    `up` or width sizes are filled up, the filling is random too."""
    import torch
    dev = torch.device("cuda", torch.cuda.current_device())

    def normal(rows, cols, tensor_id):
        t = torch.empty((rows, cols), dtype=torch.bfloat16, device=dev)
        rc = lib().vx_b200_fill_normal(t.data_ptr(), 1, t.numel(),
                                       seed * 1000003 + tensor_id, sigma)
        assert rc == 0, lib().vx_b200_last_error()
        return t

    ones = torch.ones(config.dim, dtype=torch.float32, device=dev)
    turns = torch.from_numpy(turns_per_position(config.width)).to(dev)
    embed = normal(config.vocab_rows, config.dim, 1)
    keep, owned = [ones, turns, embed], {}
    for i, s in enumerate(config.layers):
        if s.source == i:
            pair = (normal(s.in_rows, config.dim, 16 * (i + 1)),
                    normal(config.dim, s.out_cols, 16 * (i + 1) + 1))
            keep.append(pair)
            owned[i] = (ones.data_ptr(), pair[0].data_ptr(), pair[1].data_ptr())
    torch.cuda.synchronize()
    tensors = dict(layers=owned, embed=embed.data_ptr(), embed_norm=ones.data_ptr(),
                   final_norm=ones.data_ptr(), turns=turns.data_ptr())
    return decoder_of(config, tensors, True, max_seq, batch, prefill_rows, keep)
