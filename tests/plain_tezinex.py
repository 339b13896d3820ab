"""A plain, slow implementation of the Tezinex design in float64 on the CPU, one function per mechanism, written from
the design's equations and sharing no code with the library.

Notation: x the residual stream [tokens, width]; a layer computes x += m norm1b(mixer(norm1(x))) and, where it has a
feed-forward, x += m norm2b(ff(norm2(x))), m one number of the model; with X_0 the embedding's output and X_(i+1) what
layer i computes, the stream that leaves layer i is the weighted sum of X_0 .. X_(i+1). Positions count from 0 in each
sequence. A sequence's state is, per layer, what its mixer keeps of earlier positions."""
from __future__ import annotations

import math

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def zero_centred_norm(x, w, eps):
    return rms(x, eps) * (1.0 + w)


def sinusoid(positions, width):
    """[positions, width]: entry 2i is sin(p f_i), entry 2i + 1 cos(p f_i), f_i = 10000^(-2i / width)."""
    i = np.arange(width) // 2
    angles = np.asarray(positions, dtype=np.float64)[:, None] * (10000.0 ** (-2.0 * i / width))[None, :]
    return np.where(np.arange(width)[None, :] % 2 == 0, np.sin(angles), np.cos(angles))


def cap(z, limit):
    return z if limit is None else limit * np.tanh(z / limit)


def short_convolution(x, taps, history):
    """Causal convolution over time per channel: y_t = sum_j taps[:, j] x_(t - (n - 1) + j), the last tap on the token
    itself; `history` [n - 1, channels] are the inputs before x. Returns y and the new history."""
    n = taps.shape[1]
    line = np.concatenate([history, x])
    y = sum(taps[:, j][None, :] * line[j:j + len(x)] for j in range(n))
    return y, line[len(line) - (n - 1):]


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def channel_decay(w, m, h):
    """The factor of every head's key channels: exp(-exp(A_log) softplus(W_a2 W_a1 h + dt_bias)) [tokens, heads, dim]."""
    z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
    z = softplus(z).reshape(len(h), m["heads"], m["dim"])
    return np.exp(-np.exp(w["A_log"])[None, :, None] * z)


def delta_scan(q, k, v, g, beta, state):
    """Per head, token by token: the state's rows shrink, what the state already answers to k is taken off v, the rest
    is written, and the read-out sees the write. q, k, g [tokens, heads, dim], v [tokens, heads, vdim], beta [tokens,
    heads], state [heads, dim, vdim] (moved on in place)."""
    out = np.zeros(v.shape)
    for t in range(len(q)):
        state *= g[t][:, :, None]
        answer = np.einsum("hdv,hd->hv", state, k[t])
        u = beta[t][:, None] * (v[t] - answer)
        state += k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", state, q[t])
    return out


def channel_delta(w, m, h, kept, eps):
    """h [tokens, width] of ONE sequence; `kept` = {state, one convolution history for q, k and v each} (None at the
    start)."""
    heads, groups, dim, vdim, taps = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
    n = len(h)
    if kept is None:
        kept = {"S": np.zeros((heads, dim, vdim)), "q": np.zeros((taps - 1, groups * dim)),
                "k": np.zeros((taps - 1, groups * dim)), "v": np.zeros((taps - 1, heads * vdim))}
    streams = {}
    new = {}
    for name in ("q", "k", "v"):
        y, new[name] = short_convolution(h @ w[name].T, w[name + ".conv"], kept[name])
        streams[name] = silu(y)
    share = heads // groups
    q = np.repeat(unit(streams["q"].reshape(n, groups, dim)) * dim ** -0.5, share, axis=1)
    k = np.repeat(unit(streams["k"].reshape(n, groups, dim)), share, axis=1)
    v = streams["v"].reshape(n, heads, vdim)
    new["S"] = kept["S"].copy()
    o = delta_scan(q, k, v, channel_decay(w, m, h), sigmoid(h @ w["b"].T), new["S"])
    o = rms(o, eps) * w["norm"]
    gate = sigmoid((h @ w["g1"].T) @ w["g2"].T)
    return (o.reshape(n, heads * vdim) * gate) @ w["o"].T, new


def visible(i, j, mask):
    """Whether position i sees position j: not ahead, and inside the window or among the first kept ones."""
    if mask is None:
        return j <= i
    return (j <= i) & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0)))


def softmax_with_sink(scores, sink):
    """scores [heads, tokens, keys] (-inf where unseen), sink [heads]: e^score over the sum of them all plus e^sink."""
    sink = np.asarray(sink, dtype=np.float64)[:, None, None]
    top = np.maximum(scores.max(axis=2, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=2, keepdims=True) + np.exp(sink - top))


def attention(w, m, h, kept, borrowed=None):
    """h [tokens, width] of ONE sequence; `kept` = (keys, values) of the positions before. A layer without keys of its
    own is given another layer's keys and values, this step's included, as `borrowed`."""
    heads, groups, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = len(h)
    q = (h @ w["q"].T + w["q.b"]).reshape(n, heads, dim)
    if borrowed is not None:
        k, v = borrowed
    else:
        k, v = h @ w["k"].T + w["k.b"], h @ w["v"].T + w["v.b"]
        if kept is not None:
            k, v = np.concatenate([kept[0], k]), np.concatenate([kept[1], v])
    total = len(k)
    share = heads // groups
    keys = np.repeat(k.reshape(total, groups, dim), share, axis=1)
    values = np.repeat(v.reshape(total, groups, vdim), share, axis=1)
    scores = cap(np.einsum("tad,sad->ats", q, keys) * m["scale"], m.get("softcap"))
    i = (total - n + np.arange(n))[:, None]
    scores = np.where(visible(i, np.arange(total)[None, :], m.get("mask"))[None], scores, -np.inf)
    weights = softmax_with_sink(scores, w["sink"])
    return np.einsum("ats,sav->tav", weights, values).reshape(n, heads * vdim) @ w["o"].T, (k, v)


def feed_forward(w, h):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def depth_average(coefficients, results):
    """The weighted sum of the embedding's output and every layer's result so far."""
    assert len(coefficients) == len(results)
    return sum(c * x for c, x in zip(coefficients, results))


def part(weights, prefix):
    return {name[len(prefix):]: np.asarray(value, dtype=np.float64) for name, value in weights.items()
            if name.startswith(prefix)}


def new_state(config):
    return [None] * len(config["layers"])


def forward(config, weights, tokens, state=None, start=0, layers_out=None):
    """Logits [tokens, vocab] of `tokens` of one sequence whose first `start` tokens are in `state`."""
    state = new_state(config) if state is None else state
    eps, m = float(config["norm"]["eps"]), float(config["residual_mult"])
    table = np.asarray(weights["embed"], dtype=np.float64)
    get = lambda name: np.asarray(weights[name], dtype=np.float64)  # noqa: E731
    x = table[np.asarray(tokens, dtype=np.int64)] + sinusoid(np.arange(start, start + len(tokens)), config["width"])
    results = [x]
    for index, layer in enumerate(config["layers"]):
        p, mixer = f"l{index}.", layer["mixer"]
        h = zero_centred_norm(x, get(p + "norm1"), eps)
        w = part(weights, p + "mix.")
        if layer["type"] == "channel_delta":
            y, state[index] = channel_delta(w, mixer, h, state[index], eps)
        elif mixer.get("kv_from") is not None:
            y, _ = attention(w, mixer, h, None, borrowed=state[mixer["kv_from"]])
        else:
            y, state[index] = attention(w, mixer, h, state[index])
        x = x + m * zero_centred_norm(y, get(p + "norm1b"), eps)
        if layer.get("mlp") is not None:
            y = feed_forward(part(weights, p + "mlp."), zero_centred_norm(x, get(p + "norm2"), eps))
            x = x + m * zero_centred_norm(y, get(p + "norm2b"), eps)
        results.append(x)
        x = depth_average(get(p + "dwa"), results)
        if layers_out is not None:
            layers_out.append(x.copy())
    return cap(zero_centred_norm(x, get("final.norm"), eps) @ table.T, config.get("logit_softcap"))


def greedy(config, weights, prompt, count):
    """The `count` tokens the model chooses greedily after `prompt`, through its own carried state."""
    state = new_state(config)
    logits = forward(config, weights, prompt, state, 0)
    out, at = [], len(prompt)
    for _ in range(count):
        out.append(int(np.argmax(logits[-1])))
        logits = forward(config, weights, [out[-1]], state, at)
        at += 1
    return out
