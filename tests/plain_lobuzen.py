"""A plain, slow restatement of the Lobuzen decoder in numpy float64, one function per mechanism.

It shares nothing with the package: it reads a config.json dictionary and a mapping tensor name ->
array, runs whole sequences from position 0 and keeps no cache.  The tests compare the engine (which
runs portions, batches and single tokens against pages) with it.

Notation: W is the model's width, T the tokens of a sequence, H query heads, G key/value heads, D the
query/key size of a head, Dv its value size, R the size of a latent.
"""

from __future__ import annotations

import math

import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, times the weight (None: no weight)."""
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


# ------------------------------------------------------------------ attention

def in_window(i, j, size):
    """Query position i sees key position j: not later, and among the last ``size`` positions, its own included
    (``size`` None: every key up to i).  Numbers or arrays."""
    return (j <= i) & (True if size is None else (i - j < size))


def softmax_rows(s, seen, sink=None):
    """Weights of the seen keys; with a sink the sum they are divided by also holds exp(sink)."""
    s = np.where(seen, s, -np.inf)
    top = s.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(s - top)
    total = e.sum(axis=-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - top)
    return e / total


def attend(q, k, v, scale, size, sinks=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] of one sequence from position 0 -> [T, H, Dv]."""
    T, H = q.shape[:2]
    G = k.shape[1]
    seen = in_window(np.arange(T)[:, None], np.arange(T)[None, :], size)
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_rows(q[:, h] @ k[:, g].T * scale, seen, None if sinks is None else sinks[h]) @ v[:, g]
    return out


def window_size(m):
    return int(m["mask"]["size"]) if m.get("mask") else None


def attention_mixer(h, w, p, m, eps):
    """h [T, W] of one sequence.  ``w``: tensors by name, ``p``: the mixer's prefix, ``m``: its entry of config.json."""
    T = h.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms_norm((h @ w[p + "q"].T).reshape(T, H, D), None, eps)
    k = rms_norm((h @ w[p + "k"].T).reshape(T, G, D), None, eps)
    v = (h @ w[p + "v"].T).reshape(T, G, Dv)
    return attend(q, k, v, float(m["scale"]), window_size(m)).reshape(T, H * Dv) @ w[p + "o"].T


def latent(h, w, p, eps):
    """The latent of every position [T, R], from which keys and values are made."""
    return rms_norm(h @ w[p + "dkv"].T, w[p + "dkv.norm"], eps)


def latent_attention_mixer(h, c, w, p, m):
    """Queries from h [T, W], keys and values up-projected from the latents c [T, R] (this layer's or another's) for
    every position, head by head."""
    T = h.shape[0]
    H, D, Dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).reshape(T, H, D)
    k = (c @ w[p + "uk"].T).reshape(T, H, D)
    v = (c @ w[p + "uv"].T).reshape(T, H, Dv)
    return attend(q, k, v, float(m["scale"]), window_size(m), w[p + "sink"]).reshape(T, H * Dv) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward

def limited_dense(h, w, p, mlp):
    limit = float(mlp["limit"])
    g = np.minimum(h @ w[p + "gate"].T, limit)
    u = np.clip(h @ w[p + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def expert(x, gate, up, down):
    return (silu(x @ gate.T) * (x @ up.T)) @ down.T


def route(h, router, correction, top, groups=None):
    """Per token the chosen experts and their weights, two lists of arrays: sigmoid scores; the choice goes by score +
    correction, first among groups of neighbours (each judged by its two best), then among the experts of the groups that
    were kept; the weights are the scores themselves."""
    s = sigmoid(h @ router.T)
    chosen, weights = [], []
    for row in s:
        choice = row + correction
        if groups:
            n, keep = int(groups["count"]), int(groups["keep"])
            per = len(choice) // n
            judged = [np.sort(choice[g * per:(g + 1) * per])[::-1][:2].sum() for g in range(n)]
            kept = np.argsort(-np.array(judged), kind="stable")[:keep]
            allowed = np.zeros(len(choice), dtype=bool)
            for g in kept:
                allowed[g * per:(g + 1) * per] = True
            choice = np.where(allowed, choice, -np.inf)
        best = np.argsort(-choice, kind="stable")[:top]
        best = best[np.isfinite(choice[best])]
        chosen.append(best)
        weights.append(row[best])
    return chosen, weights


def moe(h, w, p, mlp):
    r = mlp["router"]
    chosen, weights = route(h, w[p + "router"], w[p + "correction"], int(r["top"]), r.get("groups"))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t], weights[t]):
            q = f"{p}e{e}."
            out[t] += c * expert(h[t][None], w[q + "gate"], w[q + "up"], w[q + "down"])[0]
    return out


FEED_FORWARDS = {"dense": limited_dense, "moe": moe}


# ------------------------------------------------------------------ a token's own input to every layer

def token_input(x, rows, w, p, eps):
    """rows [T, dim]: the tokens' vectors for this layer.  They are gated by the stream, brought to the model's width and
    normed."""
    return rms_norm((gelu_tanh(x @ w[p + "gate"].T) * rows) @ w[p + "proj"].T, w[p + "norm"], eps)


# ------------------------------------------------------------------ the model

def forward(cfg, w, tokens, keep_layers=False):
    """Logits [T, vocab] of one sequence from position 0 (and, if asked, the stream after every layer)."""
    eps = float(cfg["norm"]["eps"])
    tokens = np.asarray(tokens)
    x, after, latents = w["embed"][tokens], [], {}
    side = int((cfg.get("token_side") or {}).get("dim") or 0)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        if layer["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                latents[i] = latent(x, w, p + "mix.", eps)
            y = latent_attention_mixer(x, latents[i if src is None else int(src)], w, p + "mix.", m)
        else:
            y = attention_mixer(x, w, p + "mix.", m, eps)
        x = x + rms_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            y = FEED_FORWARDS[layer["mlp"]["kind"]](x, w, p + "mlp.", layer["mlp"])
            x = x + rms_norm(y, w[p + "norm2"], eps)
        if side:
            x = x + token_input(x, w["side.embed"][tokens, i * side:(i + 1) * side], w, p + "side.", eps)
        after.append(x.copy())
    z = rms_norm(x, w["final.norm"], eps) @ w["embed"].T
    return (z, after) if keep_layers else z
