"""A plain restatement of the Vamalix decoder in numpy, float64 throughout, one
function per mechanism: what the tests compare the GPU decoder with.  It is
written from the equations alone, token by token where that is clearest, keeps no
cache, and shares no code with vx_b200.

A model is a dict of float64 arrays by tensor name and the parsed config.
"""
import math

import numpy as np


def rms_norm(x, w, eps):
    """The last axis over sqrt(its mean square + eps), times w."""
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * w


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def gelu(z):
    """z times the normal distribution function of z."""
    phi = np.vectorize(lambda v: 0.5 * math.erfc(-v / math.sqrt(2.0)))
    return z * phi(z) if z.size else z


def rotate(x, p, base):
    """The pairs (2i, 2i + 1) of the last axis turned by p base^(-2i / n)."""
    n = x.shape[-1]
    out = np.empty_like(x)
    for i in range(n // 2):
        angle = p * float(base) ** (-2.0 * i / n)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * math.cos(angle) - v * math.sin(angle)
        out[..., 2 * i + 1] = v * math.cos(angle) + u * math.sin(angle)
    return out


def sees(i, j, window):
    """Whether the token at position i attends the one at position j."""
    return 0 <= i - j < window


def softmax(scores):
    e = np.exp(scores - scores.max())
    return e / e.sum()


def latent_attention(h, first, weights, name, m, eps):
    """h [T, width] at positions first ..: queries, keys and values out of two
    latents, one rotated key part for all heads, a sliding window."""
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    t = lambda part: weights[name + ".mix." + part]
    q = rms_norm(h @ t("dq").T, t("dq.norm"), eps) @ t("uq").T
    q = q.reshape(T, H, D + R)
    down = h @ t("dkv").T
    c = rms_norm(down[:, :K], t("dkv.norm"), eps)
    k = (c @ t("uk").T).reshape(T, H, D)
    v = (c @ t("uv").T).reshape(T, H, V)
    base = m["rot"]["base"]
    q_rot = np.stack([rotate(q[i, :, D:], first + i, base) for i in range(T)])
    k_rot = np.stack([rotate(down[i, K:], first + i, base) for i in range(T)])
    out = np.zeros((T, H, V))
    for i in range(T):
        seen = [j for j in range(max(0, i - m["mask"]["size"] - 1), T)
                if sees(i, j, m["mask"]["size"])]
        for a in range(H):
            s = (k[seen, a] @ q[i, a, :D] + k_rot[seen] @ q_rot[i, a]) * m["scale"]
            out[i, a] = softmax(s) @ v[seen, a]
    return out.reshape(T, H * V) @ t("o").T


def decays(h, weights, name, tau):
    """sigmoid(z)^(1 / tau) per key channel, z through a narrow middle."""
    z = h @ weights[name + ".mix.a1"].T @ weights[name + ".mix.a2"].T
    return sigmoid(z + weights[name + ".mix.a2.b"]) ** (1.0 / tau)


def recurrence(q, k, v, alpha, state=None):
    """State [D, V] of one head: its rows fade by alpha, k v^T comes in, q reads.
    q, k, alpha [T, D], v [T, V]; returns (o [T, V], state)."""
    state = np.zeros((q.shape[1], v.shape[1])) if state is None else state
    out = np.empty_like(v)
    for i in range(len(q)):
        state = alpha[i][:, None] * state + np.outer(k[i], v[i])
        out[i] = q[i] @ state
    return out, state


def gated_linear_attention(h, weights, name, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    t = lambda part: weights[name + ".mix." + part]
    q = (h @ t("q").T).reshape(T, H, D) / math.sqrt(D)
    k = (h @ t("k").T).reshape(T, H, D)
    v = (h @ t("v").T).reshape(T, H, V)
    alpha = decays(h, weights, name, m["tau"]).reshape(T, H, D)
    o = np.stack([recurrence(q[:, a], k[:, a], v[:, a], alpha[:, a])[0]
                  for a in range(H)], axis=1)
    o = rms_norm(o, t("norm"), eps).reshape(T, H * V)
    g = h @ t("g").T
    return (o * g * sigmoid(g)) @ t("o").T


def feed_forward(h, weights, name):
    return gelu(h @ weights[name + ".mlp.up"].T) @ weights[name + ".mlp.down"].T


def mixed_streams(x, y, mix, out):
    """x [streams, T, width]: every stream anew from all the old ones (mix is
    [from, to]) and the sublayer's output."""
    new = np.empty_like(x)
    for t in range(x.shape[0]):
        new[t] = out[t] * y
        for s in range(x.shape[0]):
            new[t] += mix[s, t] * x[s]
    return new


def sublayer(x, weights, name, q, norm, eps, f):
    """What sublayer q (1 or 2) of a layer does to the streams."""
    t = lambda part: weights["%s.hc%d.%s" % (name, q, part)]
    u = sum(t("in")[s] * x[s] for s in range(x.shape[0]))
    y = f(rms_norm(u, weights["%s.norm%d" % (name, norm)], eps))
    return mixed_streams(x, y, t("mix"), t("out"))


def layer(x, first, weights, config, i):
    name, entry, eps = "l%d" % i, config["layers"][i], config["norm"]["eps"]
    m = entry["mixer"]
    if entry["type"] == "latent_attention":
        mixer = lambda h: latent_attention(h, first, weights, name, m, eps)
    else:
        mixer = lambda h: gated_linear_attention(h, weights, name, m, eps)
    x = sublayer(x, weights, name, 1, 1, eps, mixer)
    if entry.get("mlp") is not None:
        x = sublayer(x, weights, name, 2, 2, eps,
                     lambda h: feed_forward(h, weights, name))
    return x


def order(config):
    """The layers in the order they run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + \
        list(range(loop["stop"], n))


def streams(tokens, weights, config, first=0):
    """The streams after every layer run, a list of [streams, T, width]."""
    x = weights["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    x = np.stack([x] * config["streams"])
    stages = []
    for i in order(config):
        x = layer(x, first, weights, config, i)
        stages.append(x)
    return stages


def logits(tokens, weights, config, first=0):
    x = streams(tokens, weights, config, first)[-1].sum(axis=0)
    z = rms_norm(x, weights["final.norm"], config["norm"]["eps"]) @ weights["head"].T
    cap = config["logit_softcap"]
    return cap * np.tanh(z * config["logit_scale"] / cap)


def greedy(prompt, n, weights, config):
    """n tokens after the prompt, each the largest logit (the lowest index of
    equals), the whole sequence computed afresh for every one."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(np.argmax(logits(tokens, weights, config)[-1])))
    return tokens[len(prompt):]
