"""A plain restatement of the Gofilorn decoder in numpy, float64 throughout, one
function per mechanism: what the tests compare the GPU decoder with.  It is
written from the equations alone, loops where loops are clearest, keeps no
cache, and shares no code with vx_b200.

A model is a dict of float64 arrays by tensor name and the parsed config.
"""
import numpy as np


def rms_norm(x, w, eps):
    """Each row of x over sqrt(its mean square + eps), times the gain 1 + w."""
    out = np.empty_like(x)
    for t in range(x.shape[0]):
        mean_square = float((x[t] * x[t]).sum()) / x.shape[1]
        out[t] = x[t] / np.sqrt(mean_square + eps) * (1.0 + w)
    return out


def position_vector(p, width):
    """sin(p f_i) at 2i and cos(p f_i) at 2i + 1, f_i = 10000^(-2i / width)."""
    v = np.empty(width)
    for c in range(width):
        i = c // 2
        angle = p * 10000.0 ** (-2.0 * i / width)
        v[c] = np.sin(angle) if c % 2 == 0 else np.cos(angle)
    return v


def embed(tokens, first, table, scale, gain, eps):
    """Scaled embedding rows, plus the position vector, through a norm."""
    x = np.stack([table[tok] * scale + position_vector(first + t, table.shape[1])
                  for t, tok in enumerate(tokens)])
    return rms_norm(x, gain, eps)


def sees(i, j, window):
    """Whether the token at position i attends the one at position j."""
    return 0 <= i - j < window


def softmax(scores):
    e = np.exp(scores - scores.max())
    return e / e.sum()


def attention(q, k, window, scale):
    """q [T, H, D] over k [T, G, D], the keys being the values as well; query
    head h reads key head h // (H / G). Scores are plain scaled products."""
    T, H, D = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, D))
    for i in range(T):
        seen = [j for j in range(T) if sees(i, j, window)]
        for h in range(H):
            keys = k[seen, h // (H // G)]
            out[i, h] = softmax(keys @ q[i, h] * scale) @ keys
    return out


def gate(h, w):
    return 1.0 / (1.0 + np.exp(-(h @ w.T)))


def mixer(h, weights, name, m):
    """The attention sublayer of h [T, width], gated before the output matrix."""
    T = h.shape[0]
    q = (h @ weights[name + ".mix.q"].T).reshape(T, m["heads"], m["dim"])
    k = (h @ weights[name + ".mix.k"].T).reshape(T, m["kv_heads"], m["dim"])
    a = attention(q, k, m["mask"]["size"], m["scale"]).reshape(T, -1)
    a = a * gate(h, weights[name + ".mix.g"])
    return a @ weights[name + ".mix.o"].T


def feed_forward(h, weights, name):
    """W_down relu(W_up h)^2."""
    u = np.maximum(h @ weights[name + ".mlp.up"].T, 0.0)
    return (u * u) @ weights[name + ".mlp.down"].T


def owner(layers, i):
    """The layer whose tensors layer i uses."""
    while "weights_of" in layers[i]:
        i = layers[i]["weights_of"]
    return i


def layer(x, weights, config, i):
    """Both sublayers read one norm of x, and their sum is added to x."""
    name = "l%d" % owner(config["layers"], i)
    entry = config["layers"][i]
    h = rms_norm(x, weights[name + ".norm1"], config["norm"]["eps"])
    change = mixer(h, weights, name, entry["mixer"])
    if entry.get("mlp") is not None:
        change = change + feed_forward(h, weights, name)
    return x + change


def residuals(tokens, weights, config):
    """The residual stream after every layer, [layers, T, width]."""
    x = embed(tokens, 0, weights["embed"], config["embedding"]["scale"],
              weights["embed.norm"], config["norm"]["eps"])
    stages = []
    for i in range(len(config["layers"])):
        x = layer(x, weights, config, i)
        stages.append(x)
    return np.stack(stages)


def logits(tokens, weights, config):
    """[T, vocab]: the classifier is the embedding matrix, unscaled."""
    x = residuals(tokens, weights, config)[-1]
    return rms_norm(x, weights["final.norm"], config["norm"]["eps"]) @ weights["embed"].T


def greedy(prompt, n, weights, config):
    """n tokens after the prompt, each the largest logit (the lowest index of
    equals), the whole sequence computed afresh for every one."""
    tokens = list(prompt)
    for _ in range(n):
        tokens.append(int(np.argmax(logits(tokens, weights, config)[-1])))
    return tokens[len(prompt):]
