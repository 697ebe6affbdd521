"""A plain, slow restatement of the Zatusun decoder in numpy float64, one function per mechanism.

It shares nothing with the package: it reads a config.json dictionary and a mapping tensor name ->
array, runs whole sequences from position 0 and keeps no cache.  The tests compare the engine (which
runs portions, batches and single tokens against pages and state slots) with it.

Notation: W is the model's width, T the tokens of a sequence, H query heads, G key/value heads, D the
query/key size of a head, Dv its value size.
"""

from __future__ import annotations

import math

import numpy as np


def sigmoid(x):
    return 1.0 / (1.0 + np.exp(-x))


def silu(x):
    return x * sigmoid(x)


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis, times the weight (None: no weight)."""
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def centred_rms_norm(x, weight, eps):
    """The norm in front of the sublayers and of the head: its stored weight is the factor minus one."""
    return rms_norm(x, 1.0 + weight, eps)


def soft_cap(x, cap):
    return cap * np.tanh(x / cap)


# ------------------------------------------------------------------ rotation

def plain_frequencies(dims, base):
    return np.array([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=np.float64)


def ramped_frequencies(dims, base, factor, original, fast, slow):
    """(frequencies, factor on cos and sin): pair i's frequency goes from f_i to f_i / factor along a ramp over the pair
    index, which starts at the pair that turns ``fast`` times over the original length and ends at the one that turns
    ``slow`` times."""
    f = plain_frequencies(dims, base)

    def pair_of(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    first, last = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
    for i in range(len(f)):
        ramp = min(1.0, max(0.0, (i - first) / max(last - first, 0.001)))
        f[i] = f[i] * (1.0 - ramp) + f[i] / factor * ramp
    return f, 1.0 + 0.1 * math.log(factor)


def banded_frequencies(dims, base, factor, low, high, original):
    """Frequencies by wavelength: waves shorter than original / high stay, waves longer than original / low are
    divided by ``factor``, and in between the two are blended."""
    f = plain_frequencies(dims, base)
    for i in range(len(f)):
        wave = 2.0 * math.pi / f[i]
        if wave > original / low:
            f[i] /= factor
        elif not wave < original / high:
            s = (original / wave - low) / (high - low)
            f[i] = (1.0 - s) * f[i] / factor + s * f[i]
    return f


def rotate_pairs(x, positions, freqs, grow=1.0):
    """x [T, ..., D]: neighbouring channels 2i, 2i + 1 turn by the angle position * freqs[i] and grow by ``grow``;
    channels behind the last pair pass."""
    out = x.copy()
    pos = np.asarray(list(positions), dtype=np.float64).reshape((-1,) + (1,) * (x.ndim - 2))
    for i, f in enumerate(freqs):
        c, s = np.cos(pos * f) * grow, np.sin(pos * f) * grow
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------ attention

def softmax_rows(s, seen):
    s = np.where(seen, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def same_block(i, j, size):
    """Query position i sees key position j: not later, and in the same block of ``size`` positions counted from 0."""
    return (j <= i) & (True if size is None else (i // size == j // size))       # numbers or arrays


def difference_weight(w, p, diff):
    return math.exp(float(np.sum(w[p + "lq1"] * w[p + "lk1"]))) - math.exp(float(np.sum(w[p + "lq2"] * w[p + "lk2"]))) + diff


def two_map_attention(q, k, v, scale, size, lam, diff, eps):
    """q [T, H, 2, D], k [T, G, 2, D], v [T, G, Dv] of one sequence from position 0 -> [T, H, Dv]: the second map's
    result times ``lam`` is taken from the first's, and each head's difference is divided by its root mean square."""
    T, H = q.shape[:2]
    G = k.shape[1]
    seen = same_block(np.arange(T)[:, None], np.arange(T)[None, :], size)
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        g = h // (H // G)
        a = [softmax_rows(q[:, h, m] @ k[:, g, m].T * scale, seen) @ v[:, g] for m in (0, 1)]
        out[:, h] = rms_norm(a[0] - lam * a[1], None, eps) * (1.0 - diff)
    return out


def attention_mixer(h, w, p, m, eps):
    """h [T, W] of one sequence.  ``w``: tensors by name, ``p``: the mixer's prefix, ``m``: its entry of config.json."""
    T = h.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w[p + "q"].T).reshape(T, H, 2, D)
    k = (h @ w[p + "k"].T).reshape(T, G, 2, D)
    v = (h @ w[p + "v"].T).reshape(T, G, Dv)
    rot = m.get("rot")
    if rot and int(rot["dims"]):
        sc = rot.get("scaling")
        args = (int(rot["dims"]), float(rot["base"]))
        f = banded_frequencies(*args, sc["factor"], sc["low"], sc["high"], sc["original"]) if sc else plain_frequencies(*args)
        q, k = rotate_pairs(q, range(T), f), rotate_pairs(k, range(T), f)
    size = int(m["mask"]["size"]) if m.get("mask") else None
    diff = float(m["diff"])
    a = two_map_attention(q, k, v, float(m["scale"]), size, difference_weight(w, p, diff), diff, eps)
    return a.reshape(T, H * Dv) @ w[p + "o"].T


def latent_attention_mixer(h, w, p, m, eps):
    """Queries, keys and values from low-rank latents; one turned key part for all heads; a sigmoid gate on the result.
    Keys and values are up-projected here for every position, head by head."""
    T = h.shape[0]
    H, D, R, Dv, rank = (int(m[n]) for n in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, D + R)
    d = h @ w[p + "dkv"].T
    c, k_turned = rms_norm(d[:, :rank], w[p + "dkv.norm"], eps), d[:, rank:]
    q_turned = q[:, :, D:]
    rot = m.get("rot")
    if R and rot:
        args, sc = (int(rot["dims"]), float(rot["base"])), rot.get("scaling")
        f, grow = (ramped_frequencies(*args, sc["factor"], sc["original"], sc["fast"], sc["slow"]) if sc
                   else (plain_frequencies(*args), 1.0))
        q_turned, k_turned = rotate_pairs(q_turned, range(T), f, grow), rotate_pairs(k_turned, range(T), f, grow)
    k = (c @ w[p + "uk"].T).reshape(T, H, D)
    v = (c @ w[p + "uv"].T).reshape(T, H, Dv)
    seen = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, Dv))
    for a in range(H):
        s = (q[:, a, :D] @ k[:, a].T + q_turned[:, a] @ k_turned.T) * float(m["scale"])
        out[:, a] = softmax_rows(s, seen) @ v[:, a]
    gated = out.reshape(T, H * Dv) * sigmoid(h @ w[p + "g"].T)
    return gated @ w[p + "o"].T


# ------------------------------------------------------------------ recurrence

def decayed_memory(q, f, v):
    """One head of one sequence from an empty memory: q, f [T, N], v [T, Dv].  Row n of the memory [N, Dv] decays by
    f_t[n] and takes (1 - f_t[n]) v_t."""
    S = np.zeros((q.shape[1], v.shape[1]))
    out = np.zeros((q.shape[0], v.shape[1]))
    for t in range(q.shape[0]):
        S = f[t][:, None] * S + (1.0 - f[t])[:, None] * v[t][None, :]
        out[t] = q[t] @ S
    return out


def hgrn2_mixer(h, w, p, m, eps):
    T = h.shape[0]
    H, N, Dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ w[p + "q"].T).reshape(T, H, N)
    low = w[p + "lower"]
    f = (low + (1.0 - low) * sigmoid(h @ w[p + "f"].T + w[p + "f.b"])).reshape(T, H, N)
    v = (h @ w[p + "v"].T).reshape(T, H, Dv)
    o = np.stack([decayed_memory(q[:, a], f[:, a], v[:, a]) for a in range(H)], axis=1)
    return rms_norm(o, w[p + "norm"], eps).reshape(T, H * Dv) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward

def limited_expert(x, gate, up, down, limit):
    """x [T, W] -> [T, W]: g = min(gate x, limit), u = clamp(up x, -limit, limit), down (g sigmoid(1.702 g) (u + 1))."""
    g = np.minimum(x @ gate.T, limit)
    u = np.clip(x @ up.T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ down.T


def route(h, router, top):
    """(chosen expert indices [T, top], their weights [T, top]): the largest logits, softmax over those alone."""
    z = h @ router.T
    order = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    e = np.take_along_axis(z, order, axis=-1)
    e = np.exp(e - e.max(axis=-1, keepdims=True))
    return order, e / e.sum(axis=-1, keepdims=True)


def moe(h, w, p, mlp):
    chosen, weight = route(h, w[p + "router"], int(mlp["router"]["top"]))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(chosen[t], weight[t]):
            q = f"{p}e{e}."
            out[t] += c * limited_expert(h[t][None], w[q + "gate"], w[q + "up"], w[q + "down"],
                                         float(mlp["expert"]["limit"]))[0]
    return out


# ------------------------------------------------------------------ the model

def embed(cfg, w, tokens):
    return w["embed"][np.asarray(tokens)] * float(cfg["embedding"]["scale"]) + w["pos"][:len(tokens)]


def layer_runs(cfg):
    """(layer, number of the pass that this run opens or None), in the order in which they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = int(loop["start"]), int(loop["stop"])
    runs = [(i, None) for i in range(a)]
    for t in range(int(loop["times"])):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def start_pass(x, x0, w, t):
    """What stands in front of pass t's first layer: a product over the stream and the embedding's output side by
    side, and the pass's vector."""
    return np.concatenate([x, x0], axis=-1) @ w["loop.in"].T + w["loop.step"][t]


MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer, "hgrn2": hgrn2_mixer}


def forward(cfg, w, tokens, keep_layers=False):
    """Logits [T, vocab] of one sequence from position 0 (and, if asked, the stream after every layer run)."""
    eps = float(cfg["norm"]["eps"])
    x0 = embed(cfg, w, tokens)
    x, after = x0, []
    for i, opens in layer_runs(cfg):
        p, layer = f"l{i}.", cfg["layers"][i]
        if opens is not None:
            x = start_pass(x, x0, w, opens)
        x = x + MIXERS[layer["type"]](centred_rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + moe(centred_rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", layer["mlp"])
        after.append(x.copy())
    z = centred_rms_norm(x, w["final.norm"], eps) @ w["head"].T
    if cfg.get("logit_softcap"):
        z = soft_cap(z, float(cfg["logit_softcap"]))
    return (z, after) if keep_layers else z
