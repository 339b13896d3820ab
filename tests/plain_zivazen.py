"""A plain, slow implementation of the Zivazen design in float64 on the CPU, one function per mechanism, written from
the design's equations and sharing no code with the library.

Notation: x the residual stream [tokens, width], which starts as the normed embedding rows; a layer computes
x += mixer(h) + ff(h) with ONE h = norm1(x) for both (a layer may have no ff). Positions count from 0 in each sequence.
A sequence's state is, per layer, what its mixer keeps of earlier positions."""
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


def linear(w, name, h):
    """h through the matrix `name`, plus the bias `name.b` where the weights have one."""
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


# ---- rotation -----------------------------------------------------------------------------------------------------------


def frequencies(rot):
    """One per rotated pair; with `scaling`, long wavelengths are stretched by the factor, short ones stay, and those
    between are joined linearly in original / wavelength."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s is not None:
            wavelength = 2 * math.pi / f
            if wavelength > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wavelength >= s["original"] / s["high"]:
                t = (s["original"] / wavelength - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return np.array(out)


def rotate(x, positions, rot):
    """x [tokens, heads, dim]: dimension i turns with i + dims / 2 by position times frequency; the rest stays."""
    if not rot or not rot["dims"]:
        return x
    half = rot["dims"] // 2
    a = np.asarray(positions, dtype=np.float64)[:, None, None] * frequencies(rot)[None, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a), x[..., 2 * half:]], axis=-1)


# ---- attention ----------------------------------------------------------------------------------------------------------


def same_chunk(i, j, size):
    return (j <= i) & (i // size == j // size)


def in_window(i, j, size):
    return (j <= i) & (i - j < size)


def softmax_plus_one(scores):
    """e^s over one plus their sum: scores [..., keys], -inf where unseen."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), 0.0)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(-top))


def softmax(scores):
    e = np.exp(scores - scores.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def attend(q, k, v, scale, seen, normalise):
    """q [n, heads, dim] at the last n of the positions of k [m, groups, dim] and v [m, groups, vdim]; `seen(i, j)` the
    mask, `normalise` the softmax."""
    n, heads, m, groups = len(q), q.shape[1], len(k), k.shape[1]
    keys, values = np.repeat(k, heads // groups, axis=1), np.repeat(v, heads // groups, axis=1)
    scores = np.einsum("tad,sad->ats", q, keys) * scale
    i = (m - n + np.arange(n))[:, None]
    scores = np.where(seen(i, np.arange(m)[None, :])[None], scores, -np.inf)
    return np.einsum("ats,sav->tav", normalise(scores), values).reshape(n, -1)


def mix_values(v, first, share):
    return (1 - share) * v + share * first


def attention(w, m, h, kept, start, eps, values):
    """Keys and queries normed per head and turned, chunks, a softmax with one more in its denominator. `values` [0] holds
    what the step's first layer of those that mix values projected (set by it, read by the others)."""
    n = len(h)
    positions = np.arange(start, start + n)
    q = linear(w, "q", h).reshape(n, m["heads"], m["dim"])
    k = linear(w, "k", h).reshape(n, m["kv_heads"], m["dim"])
    v = linear(w, "v", h).reshape(n, m["kv_heads"], m["vdim"])
    q = rotate(rms(q, eps) * w["q.norm"], positions, m.get("rot"))
    k = rotate(rms(k, eps) * w["k.norm"], positions, m.get("rot"))
    if m.get("v_mix"):
        if not values:
            values.append(v)
        else:
            v = mix_values(v, values[0], float(w["vmix"]))
    if kept is not None:
        k, v = np.concatenate([kept[0], k]), np.concatenate([kept[1], v])
    mask = m.get("mask")
    seen = (lambda i, j: j <= i) if mask is None else (lambda i, j: same_chunk(i, j, mask["size"]))
    return linear(w, "o", attend(q, k, v, m["scale"], seen, softmax_plus_one)), (k, v)


def windowed_attention(w, m, h, kept, start):
    n = len(h)
    positions = np.arange(start, start + n)
    q = rotate(linear(w, "q", h).reshape(n, m["heads"], m["dim"]), positions, m.get("rot"))
    k = rotate(linear(w, "k", h).reshape(n, m["kv_heads"], m["dim"]), positions, m.get("rot"))
    v = linear(w, "v", h).reshape(n, m["kv_heads"], m["vdim"])
    if kept is not None:
        k, v = np.concatenate([kept[0], k]), np.concatenate([kept[1], v])
    mask = m.get("mask")
    seen = (lambda i, j: j <= i) if mask is None else (lambda i, j: in_window(i, j, mask["size"]))
    return linear(w, "o", attend(q, k, v, m["scale"], seen, softmax)), (k, v)


# ---- state-space branch -------------------------------------------------------------------------------------------------


def short_convolution(x, taps, bias, history):
    """Causal, per channel: y_t = bias + sum_j taps[:, j] x_(t - (n - 1) + j); `history` [n - 1, channels] the inputs before
    x. Returns y and the new history."""
    n = taps.shape[1]
    line = np.concatenate([history, x])
    y = bias + sum(taps[:, j][None, :] * line[j:j + len(x)] for j in range(n))
    return y, line[len(line) - (n - 1):]


def state_space_scan(x, b, c, dt, rate, skip, state):
    """Token by token per head: S <- exp(-rate dt) S + dt b x^T, y = S^T c + skip x. x [n, heads, vdim], b and c [n, heads,
    N], dt [n, heads], rate and skip [heads], state [heads, N, vdim] (moved on in place)."""
    y = np.zeros(x.shape)
    for t in range(len(x)):
        state *= np.exp(-rate * dt[t])[:, None, None]
        state += dt[t][:, None, None] * b[t][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnv,hn->hv", state, c[t]) + skip[:, None] * x[t]
    return y


def gate_then_norm(y, z, weight, parts, eps):
    gated = y * silu(z)
    n, inner = gated.shape
    return rms(gated.reshape(n, parts, inner // parts), eps).reshape(n, inner) * weight


def state_space(w, m, h, kept, eps):
    heads, vdim, size, groups, taps = m["heads"], m["vdim"], m["state"], m["groups"], m["conv"]
    inner, n = heads * vdim, len(h)
    channels = inner + 2 * groups * size
    if kept is None:
        kept = (np.zeros((heads, size, vdim)), np.zeros((taps - 1, channels)))
    u = h @ w["in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:inner + channels], u[:, inner + channels:]
    xbc, history = short_convolution(xbc, w["conv"], w["conv.b"], kept[1])
    xbc = silu(xbc)
    x = xbc[:, :inner].reshape(n, heads, vdim)
    share = heads // groups
    b = np.repeat(xbc[:, inner:inner + groups * size].reshape(n, groups, size), share, axis=1)
    c = np.repeat(xbc[:, inner + groups * size:].reshape(n, groups, size), share, axis=1)
    state = kept[0].copy()
    y = state_space_scan(x, b, c, softplus(dt + w["dt_bias"]), np.exp(w["A_log"]), w["D"], state)
    return gate_then_norm(y.reshape(n, inner), z, w["norm"], m["norm_groups"], eps) @ w["o"].T, (state, history)


def parallel(w, m, h, kept, start, eps):
    kept = (None, None) if kept is None else kept
    left, kept_left = windowed_attention(part(w, "left."), m["left"], h, kept[0], start)
    right, kept_right = state_space(part(w, "right."), m["right"], h, kept[1], eps)
    return m["left_scale"] * left + m["right_scale"] * right, (kept_left, kept_right)


# ---- feed-forward -------------------------------------------------------------------------------------------------------


def dense(w, h):
    return linear(w, "down", silu(linear(w, "gate", h)) * linear(w, "up", h))


def squared_relu_unit(w, h):
    return np.maximum(h @ w["up"].T, 0.0) ** 2 @ w["down"].T


def choose(scores, correction, router):
    """One token's experts: the `top` largest of scores + correction inside the `keep` groups of neighbours whose two
    largest add up to the most. Their weights: the plain scores over their sum, times the router's scale."""
    choice = scores + correction
    groups = router.get("groups")
    if groups is not None:
        size = len(scores) // groups["count"]
        totals = [np.sort(choice[g * size:(g + 1) * size])[-2:].sum() for g in range(groups["count"])]
        best = np.argsort(-np.array(totals), kind="stable")[:groups["keep"]]
        open_ = np.isin(np.arange(len(scores)) // size, best)
        choice = np.where(open_, choice, -np.inf)
    picked = np.argsort(-choice, kind="stable")[:router["top"]]
    return picked, scores[picked] / (scores[picked].sum() + 1e-20) * router["scale"]


def mixture(w, mlp, h):
    scores = sigmoid(h @ w["router"].T)
    out = np.zeros_like(h)
    for t in range(len(h)):
        for expert, weight in zip(*choose(scores[t], w["correction"], mlp["router"])):
            out[t] += weight * squared_relu_unit(part(w, f"e{expert}."), h[t])
    if mlp.get("shared") is not None:
        out += squared_relu_unit(part(w, "shared."), h)
    return out


# ---- the model ----------------------------------------------------------------------------------------------------------


def part(weights, prefix):
    return {name[len(prefix):]: np.asarray(value, dtype=np.float64) for name, value in weights.items()
            if name.startswith(prefix)}


def new_state(config):
    return [None] * len(config["layers"])


def forward(config, weights, tokens, state=None, start=0, layers_out=None):
    """Logits [tokens, vocab] of `tokens` of one sequence whose first `start` tokens are in `state`."""
    state = new_state(config) if state is None else state
    eps = float(config["norm"]["eps"])
    get = lambda name: np.asarray(weights[name], dtype=np.float64)  # noqa: E731
    x = rms(get("embed")[np.asarray(tokens, dtype=np.int64)], eps) * get("embed.norm")
    values = []
    for index, layer in enumerate(config["layers"]):
        p = f"l{index}."
        h = rms(x, eps) * get(p + "norm1")
        w = part(weights, p + "mix.")
        if layer["type"] == "attention":
            y, state[index] = attention(w, layer["mixer"], h, state[index], start, eps, values)
        else:
            y, state[index] = parallel(w, layer["mixer"], h, state[index], start, eps)
        if layer.get("mlp") is not None:
            w = part(weights, p + "mlp.")
            y = y + (dense(w, h) if layer["mlp"]["kind"] == "dense" else mixture(w, layer["mlp"], h))
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms(x, eps) * get("final.norm") @ get("head").T


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
