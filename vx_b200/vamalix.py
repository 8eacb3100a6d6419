"""Vamalix decoders on the whole-token entry points (vx_decoder_create_streams,
include/vx_b200.h): what its config.json says, its weights in the layout of the
kernels, and synthetic models of the same architecture.

The residual is several streams; each sublayer reads a weighted sum of them and mixes
them with its output. Mixers: latent attention over a sliding window, and gated linear
attention. A run of layers may be repeated, each pass with a cache and states of its
own.
"""
import json
import math
import os

import numpy as np

from . import abi
from .lib import (MIXER_GATED_LINEAR, MIXER_LATENT, StreamConfig, StreamLayer, lib)
from .llama import Decoder
from .safetensors import SafeTensors, to_bf16

ARCHITECTURE = "Vamalix"
DTYPES = ("bfloat16", "float32")


def _up(n, step):
    return (n + step - 1) // step * step


class _Shape:
    """What both kinds of layer have: heads of `vdim` values, filled up so that a
    head is a multiple of 8 and all of them together one of 64."""

    def __init__(self, m, mlp):
        self.heads, self.dim, self.vdim = m["heads"], m["dim"], m["vdim"]
        self.head_dim = _up(self.dim, 8)
        self.head_vdim = _up(self.vdim, max(8, 64 // math.gcd(64, self.heads)))
        self.out_cols = self.heads * self.head_vdim
        self.ff = mlp["ff"] if mlp is not None else 0
        self.hidden = _up(self.ff, 64)


class LatentShape(_Shape):
    kind = MIXER_LATENT

    def __init__(self, m, mlp):
        super().__init__(m, mlp)
        self.rot, self.scale = m["rot_dim"], m["scale"]
        self.window, self.base = m["mask"]["size"], m["rot"]["base"]
        self.q_mean, self.kv_mean = m["q_rank"], m["kv_rank"]
        if m["rot"]["dims"] != self.rot or self.rot % 2:
            raise ValueError("the whole rotated part is rotated, in pairs")
        self.rot_dim = _up(self.rot, 8)
        self.q_rank, self.kv_rank = _up(self.q_mean, 64), _up(self.kv_mean, 64)
        self.in_rows = self.q_rank + self.kv_rank + self.rot_dim
        self.cache_row = self.kv_rank + self.rot_dim
        # rows of the other matrices with their columns, for counting weights
        self.inner = [(self.heads * (self.head_dim + self.rot_dim), self.q_rank),
                      (self.heads * (self.head_dim + self.head_vdim), self.kv_rank)]

    def turns(self):
        """The part of a full turn that the pair (2i, 2i + 1) advances per position."""
        out = np.zeros(max(self.rot_dim // 2, 1))
        i = np.arange(self.rot // 2, dtype=np.float64)
        if self.rot:
            out[:self.rot // 2] = float(self.base) ** (-2.0 * i / self.rot) / (2 * np.pi)
        return out


class GatedLinearShape(_Shape):
    kind = MIXER_GATED_LINEAR

    def __init__(self, m, mlp):
        super().__init__(m, mlp)
        self.tau, self.scale = m["tau"], self.dim ** -0.5
        self.k_row = self.heads * self.head_dim
        self.v_row = 2 * self.k_row
        self.gate_row = self.v_row + self.out_cols
        self.a1_row = self.gate_row + self.out_cols
        self.rank = self.a_rank = None
        self.inner = []

    def set_rank(self, rank):
        """The middle of the decays' two matrices, which only a tensor's shape says."""
        self.rank, self.a_rank = rank, _up(rank, 8)
        self.in_rows = self.a1_row + self.a_rank


MIXERS = {"latent_attention": LatentShape, "gla": GatedLinearShape}


class VamalixConfig:
    """What config.json says; `layers` holds a shape each, `order` the layers in the
    order they run."""

    def __init__(self, width, vocab, eps, embed_scale, streams, logit_scale, logit_cap,
                 layers, order):
        self.width, self.vocab, self.eps = width, vocab, eps
        self.embed_scale, self.streams = embed_scale, streams
        self.logit_scale, self.logit_cap = logit_scale, logit_cap
        self.layers, self.order = layers, order
        self.dim, self.vocab_rows = _up(width, 64), _up(vocab, 8)

    @classmethod
    def from_dict(cls, config):
        if config.get("architecture") != ARCHITECTURE:
            raise ValueError("not a %s configuration: %r"
                             % (ARCHITECTURE, config.get("architecture")))
        layers = []
        for i, entry in enumerate(config["layers"]):
            if entry.get("type") not in MIXERS:
                raise ValueError("layer %d has the type %r" % (i, entry.get("type")))
            mlp = entry.get("mlp")
            if mlp is not None and mlp.get("kind") != "dense":
                raise ValueError("layer %d has a feed-forward of the kind %r"
                                 % (i, mlp.get("kind")))
            layers.append(MIXERS[entry["type"]](entry["mixer"], mlp))
        n, loop = len(layers), config.get("loop")
        order = list(range(n))
        if loop is not None:
            start, stop, times = loop["start"], loop["stop"], loop["times"]
            if not 0 <= start <= stop <= n or times < 0:
                raise ValueError("the loop %r does not fit %d layers" % (loop, n))
            order = order[:start] + order[start:stop] * times + order[stop:]
        if not order:
            raise ValueError("no layer runs")
        return cls(config["width"], config["vocab"], config["norm"]["eps"],
                   config["embedding"]["scale"], config["streams"],
                   config["logit_scale"], config["logit_softcap"], layers, order)

    @classmethod
    def from_file(cls, path):
        with open(path) as f:
            return cls.from_dict(json.load(f))


def _filled(a, shape):
    """`a` in the corner of zeros."""
    out = np.zeros(shape, np.float32)
    out[tuple(slice(n) for n in a.shape)] = a
    return out


def pack_latent(s, width, dim, tensor):
    """The tensors of a latent-attention layer as the kernels read them, f32.
    tensor(name, shape) gives the layer's."""
    H, D, R, V = s.heads, s.dim, s.rot, s.vdim
    P, Q, U = s.head_dim, s.rot_dim, s.head_vdim
    dkv = tensor("mix.dkv", (s.kv_mean + R, width))
    w_in = np.zeros((s.in_rows, dim), np.float32)
    w_in[:s.q_mean, :width] = tensor("mix.dq", (s.q_mean, width))
    w_in[s.q_rank:s.q_rank + s.kv_mean, :width] = dkv[:s.kv_mean]
    at = s.q_rank + s.kv_rank
    w_in[at:at + R, :width] = dkv[s.kv_mean:]
    uq = tensor("mix.uq", (H * (D + R), s.q_mean)).reshape(H, D + R, s.q_mean)
    w_uq = np.zeros((H, P + Q, s.q_rank), np.float32)
    w_uq[:, :D, :s.q_mean] = uq[:, :D]
    w_uq[:, P:P + R, :s.q_mean] = uq[:, D:]
    uk = tensor("mix.uk", (H * D, s.kv_mean)).reshape(H, D, s.kv_mean)
    uv = tensor("mix.uv", (H * V, s.kv_mean)).reshape(H, V, s.kv_mean)
    w_ukv = np.zeros((H, P + U, s.kv_rank), np.float32)
    w_ukv[:, :D, :s.kv_mean] = uk
    w_ukv[:, P:P + V, :s.kv_mean] = uv
    w_uk_t = np.ascontiguousarray(w_ukv[:, :P].transpose(0, 2, 1))
    return dict(w_in=w_in, w_uq=w_uq.reshape(-1, s.q_rank),
                w_ukv=w_ukv.reshape(-1, s.kv_rank), w_uk_t=w_uk_t.reshape(-1, P),
                q_norm=_filled(tensor("mix.dq.norm", (s.q_mean,)), s.q_rank),
                kv_norm=_filled(tensor("mix.dkv.norm", (s.kv_mean,)), s.kv_rank))


def pack_gated_linear(s, width, dim, tensor):
    H, D, V, P, U = s.heads, s.dim, s.vdim, s.head_dim, s.head_vdim
    w_in = np.zeros((s.in_rows, dim), np.float32)

    def put(row, name, size, filled):
        part = w_in[row:row + H * filled, :width].reshape(H, filled, width)
        part[:, :size] = tensor(name, (H * size, width)).reshape(H, size, width)
        w_in[row:row + H * filled, :width] = part.reshape(H * filled, width)

    put(0, "mix.q", D, P)
    put(s.k_row, "mix.k", D, P)
    put(s.v_row, "mix.v", V, U)
    put(s.gate_row, "mix.g", V, U)
    w_in[s.a1_row:s.a1_row + s.rank, :width] = tensor("mix.a1", (s.rank, width))
    a2 = np.zeros((H, P, s.a_rank), np.float32)
    a2[:, :D, :s.rank] = tensor("mix.a2", (H * D, s.rank)).reshape(H, D, s.rank)
    bias = _filled(tensor("mix.a2.b", (H * D,)).reshape(H, D), (H, P))
    return dict(w_in=w_in, a2=a2.reshape(-1, s.a_rank), a2_bias=bias.reshape(-1),
                o_norm=_filled(tensor("mix.norm", (V,)), U))


def pack_layer(s, width, dim, streams, tensor):
    """All of a layer's arrays by their names in StreamLayer, f32 (hc1 and hc2 as
    triples, turns f64)."""
    out = (pack_latent if s.kind == MIXER_LATENT else pack_gated_linear)(
        s, width, dim, tensor)
    H, V, U = s.heads, s.vdim, s.head_vdim
    w_o = np.zeros((dim, H, U), np.float32)
    w_o[:width, :, :V] = tensor("mix.o", (width, H * V)).reshape(width, H, V)
    out["w_o"] = w_o.reshape(dim, -1)
    if s.kind == MIXER_LATENT:
        out["turns"] = s.turns()
    for q in (1, 2) if s.ff else (1,):
        out["norm%d" % q] = _filled(tensor("norm%d" % q, (width,)), dim)
        out["hc%d" % q] = (tensor("hc%d.in" % q, (streams,)),
                           tensor("hc%d.mix" % q, (streams, streams)),
                           tensor("hc%d.out" % q, (streams,)))
    if s.ff:
        out["w_up"] = _filled(tensor("mlp.up", (s.ff, width)), (s.hidden, dim))
        out["w_down"] = _filled(tensor("mlp.down", (width, s.ff)), (dim, s.hidden))
    return out


MATRICES = ("w_in", "w_o", "w_uq", "w_ukv", "w_uk_t", "w_up", "w_down")


def decoder_of(config, tensors, bf16, max_seq, batch=1, prefill_rows=0, keep=None):
    """A Decoder over device addresses: tensors["layers"] holds a dict of addresses by
    field name for each layer (hc1 and hc2 as triples); embed, head and final_norm are
    addresses."""
    runs = (StreamLayer * len(config.order))()
    for to, i in zip(runs, config.order):
        s = config.layers[i]
        to.kind, to.heads, to.hidden, to.scale = s.kind, s.heads, s.hidden, s.scale
        to.dim, to.vdim = s.head_dim, s.head_vdim
        if s.kind == MIXER_LATENT:
            to.rot_dim, to.window = s.rot_dim, s.window
            to.q_rank, to.q_mean = s.q_rank, s.q_mean
            to.kv_rank, to.kv_mean = s.kv_rank, s.kv_mean
        else:
            to.a_rank, to.v_mean, to.inv_tau = s.a_rank, s.vdim, 1.0 / s.tau
        for name, value in tensors["layers"][i].items():
            if name in ("hc1", "hc2"):
                mix = getattr(to, name)
                mix.hc_in, mix.mix, mix.out = value
            else:
                setattr(to, name, value)
    cfg = StreamConfig(
        width=config.width, dim=config.dim, n_layers=len(config.order),
        vocab=config.vocab, vocab_rows=config.vocab_rows, max_seq=max_seq,
        weights_bf16=1 if bf16 else 0, batch=batch, prefill_rows=prefill_rows,
        streams=config.streams, eps=config.eps, embed_scale=config.embed_scale,
        logit_scale=config.logit_scale, logit_cap=config.logit_cap or 0.0,
        embed=tensors["embed"], classifier=tensors["head"],
        final_norm=tensors["final_norm"], layers=runs)
    return Decoder.from_config(cfg, keep=(keep, runs))


def from_tensors(config, tensor, shape_of, dtype="bfloat16", max_seq=4096, batch=1,
                 prefill_rows=0):
    """A Decoder of the weights that tensor(name, shape) gives as f32; shape_of(name)
    is a tensor's shape."""
    if dtype not in DTYPES:
        raise ValueError("the dtype is one of %s" % (DTYPES,))
    bf16 = dtype == "bfloat16"
    keep = []

    def place(a):
        t = abi.DeviceTensor.from_host(np.ascontiguousarray(a))
        keep.append(t)
        return t.ptr

    def matrix(a):
        if not bf16:
            return place(a)
        t = abi.DeviceTensor.from_host(to_bf16(a), bf16=True)
        keep.append(t)
        return t.ptr

    def table(name):
        return matrix(_filled(tensor(name, (config.vocab, config.width)),
                              (config.vocab_rows, config.dim)))

    layers = {}
    for i in sorted(set(config.order)):
        s = config.layers[i]
        if s.kind == MIXER_GATED_LINEAR:
            s.set_rank(int(shape_of("l%d.mix.a1" % i)[0]))
        packed = pack_layer(s, config.width, config.dim, config.streams,
                            lambda name, shape: tensor("l%d.%s" % (i, name), shape))
        layers[i] = {name: tuple(place(p) for p in a) if name in ("hc1", "hc2")
                     else matrix(a) if name in MATRICES else place(a)
                     for name, a in packed.items()}
    tensors = dict(layers=layers, embed=table("embed"), head=table("head"),
                   final_norm=place(_filled(tensor("final.norm", (config.width,)),
                                            config.dim)))
    return decoder_of(config, tensors, bf16, max_seq, batch, prefill_rows, keep)


def load(path, dtype="bfloat16", max_seq=4096, batch=1, prefill_rows=0):
    """The model of a folder with config.json and model.safetensors."""
    config = VamalixConfig.from_file(os.path.join(path, "config.json"))
    weights = SafeTensors(os.path.join(path, "model.safetensors"))
    return from_tensors(config, weights.f32, weights.shape, dtype, max_seq, batch,
                        prefill_rows)


def synthetic(config, max_seq, rank=16, seed=7, batch=1, sigma=0.02, prefill_rows=0):
    """A bf16 model of random weights made on the GPU (torch only holds the memory):
    N(0, sigma^2) matrices, gains of 1, streams that stay near one another. For
    measurements: what fills sizes up is random too."""
    import torch
    dev = torch.device("cuda", torch.cuda.current_device())
    keep = []

    def address(t):
        keep.append(t)
        return t.data_ptr()

    def normal(rows, cols, tensor_id):
        t = torch.empty((rows, cols), dtype=torch.bfloat16, device=dev)
        rc = lib().vx_b200_fill_normal(t.data_ptr(), 1, t.numel(),
                                       seed * 1000003 + tensor_id, sigma)
        assert rc == 0, lib().vx_b200_last_error()
        return address(t)

    def full(value, *shape):
        return address(torch.full(shape, value, dtype=torch.float32, device=dev))

    S = config.streams
    mixing = (full(1.0 / S, S),
              address(0.9 * torch.eye(S, device=dev) + 0.1 / S), full(1.0, S))
    layers = {}
    for i in sorted(set(config.order)):
        s = config.layers[i]
        if s.kind == MIXER_GATED_LINEAR:
            s.set_rank(rank)
        t = dict(norm1=full(1.0, config.dim), hc1=mixing,
                 w_in=normal(s.in_rows, config.dim, 16 * (i + 1)),
                 w_o=normal(config.dim, s.out_cols, 16 * (i + 1) + 1))
        if s.kind == MIXER_LATENT:
            t.update(q_norm=full(1.0, s.q_rank), kv_norm=full(1.0, s.kv_rank),
                     turns=address(torch.from_numpy(s.turns()).to(dev)),
                     w_uq=normal(*s.inner[0], 16 * (i + 1) + 2),
                     w_ukv=normal(*s.inner[1], 16 * (i + 1) + 3))
            w = keep[-1].view(s.heads, s.head_dim + s.head_vdim, s.kv_rank)
            t["w_uk_t"] = address(w[:, :s.head_dim].transpose(1, 2).contiguous())
        else:
            t.update(a2=address(sigma * torch.randn(s.k_row, s.a_rank, device=dev)),
                     a2_bias=full(2.0, s.k_row), o_norm=full(1.0, s.head_vdim))
        if s.hidden:
            t.update(norm2=full(1.0, config.dim), hc2=mixing,
                     w_up=normal(s.hidden, config.dim, 16 * (i + 1) + 4),
                     w_down=normal(config.dim, s.hidden, 16 * (i + 1) + 5))
        layers[i] = t
    tensors = dict(layers=layers, embed=normal(config.vocab_rows, config.dim, 1),
                   head=normal(config.vocab_rows, config.dim, 2),
                   final_norm=full(1.0, config.dim))
    torch.cuda.synchronize()
    return decoder_of(config, tensors, True, max_seq, batch, prefill_rows, keep)
