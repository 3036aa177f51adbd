"""The Zomurax design restated in numpy (float64), slowly and plainly: one function per mechanism, no cache, no batch,
nothing shared with the library.  A model is a configuration (the dict of config.json) and a dict name -> array.

    tokens -> embedding rows -> layers -> final norm -> head -> cap on the logits

Every norm is an RMS norm with ONE gain for all coordinates, and stands BEHIND a branch: with a constant a,
x <- n1(a x + mixer(x)) and then x <- n2(a x + ff(x)); the branches read x itself.  A layer's mixer is either attention of
grouped queries with unit-size queries and keys, a bias that grows with the logarithm of the distance, a sink and values
that later layers mix with the first layer's, or attention through a low-rank latent over a sliding window.  The
feed-forward is a mixture of experts picked by the token's id, plus one expert that every token runs.
"""
import math

import numpy as np


# -- small pieces -----------------------------------------------------------------------------------------------------

def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def norm(x, gain, eps):
    """``gain`` is one number."""
    return rms_unit(x, eps) * float(gain)


def silu(z):
    return z / (1.0 + np.exp(-z))


def softmax(z, sink=None):
    """Weights of the scores z; ``sink`` is one more score that takes its share of the sum and stands for no key."""
    top = z.max() if sink is None else max(z.max(), sink)
    e = np.exp(z - top)
    return e / (e.sum() + (0.0 if sink is None else math.exp(sink - top)))


# -- pieces of the mixers ---------------------------------------------------------------------------------------------

def rotate_half(x, pos, base, dims):
    """x [..., head size] at position ``pos``: entry i < dims/2 turns together with entry i + dims/2 by the angle
    pos * base^(-2i/dims); entries from ``dims`` on pass."""
    y = x.copy()
    half = dims // 2
    a = pos * np.array([base ** (-2.0 * i / dims) for i in range(half)])
    c, s = np.cos(a), np.sin(a)
    u, v = x[..., :half], x[..., half:dims]
    y[..., :half] = u * c - v * s
    y[..., half:dims] = v * c + u * s
    return y


def temperature(pos, coef, every):
    """What a query at position ``pos`` is multiplied by: it grows a step every ``every`` positions."""
    return 1.0 + coef * math.log(math.floor((pos + 1) / every) + 1.0)


def distance_bias(dist, r1, r2):
    """What a key ``dist`` positions back loses of its score (``dist`` may be an array)."""
    return r1 * np.log(1.0 + r2 * dist)


def in_window(i, j, size):
    """Does the query at position i see the key at position j?  Causal; with ``size`` only itself and the size - 1 before."""
    return j <= i and (not size or i - j < size)


def mix_values(v, first, lam):
    """Whole projected rows, all heads at once."""
    return (1.0 - lam) * v + lam * first


# -- mixers -----------------------------------------------------------------------------------------------------------

def attention(m, w, p, x, eps, first_values):
    """x [tokens, width] -> (output, the layer's own values before any mixing).  ``first_values``: the values of the first
    layer that mixes, or None in that layer and in layers that do not mix."""
    H, G, dk, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    T = x.shape[0]
    q = rms_unit((x @ w[p + "q"].T).reshape(T, H, dk), eps)
    k = rms_unit((x @ w[p + "k"].T).reshape(T, G, dk), eps)
    own = x @ w[p + "v"].T
    v = (own if first_values is None else mix_values(own, first_values, float(w[p + "vmix"]))).reshape(T, G, dv)
    if m.get("q_temp"):
        q = q * np.array([temperature(t, float(m["q_temp"]["coef"]), float(m["q_temp"]["every"])) for t in range(T)])[:, None, None]
    o = np.zeros((T, H, dv))
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            s = (k[:i + 1, g] @ q[i, a]) * float(m["scale"])
            s = s - distance_bias(i - np.arange(i + 1.0), float(w[p + "r1"][a]), float(w[p + "r2"][a]))
            o[i, a] = softmax(s, float(w[p + "sink"][a])) @ v[:i + 1, g]
    return o.reshape(T, H * dv) @ w[p + "o"].T, own


def latent_attention(m, w, p, x, eps):
    """Keys and values of every head come from one normed latent per token; one rotated key part is shared by all heads."""
    H, dk, R, dv, C = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    T = x.shape[0]
    q = (x @ w[p + "q"].T).reshape(T, H, dk + R)
    down = x @ w[p + "dkv"].T
    c = rms_unit(down[:, :C], eps) * w[p + "dkv.norm"]
    r = down[:, C:]
    k = (c @ w[p + "uk"].T).reshape(T, H, dk)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    qn, qr = q[..., :dk], q[..., dk:]
    rot = m.get("rot") or {}
    if R and rot.get("dims"):
        base, dims = float(rot["base"]), int(rot["dims"])
        qr = np.stack([rotate_half(qr[t], t, base, dims) for t in range(T)])
        r = np.stack([rotate_half(r[t], t, base, dims) for t in range(T)])
    size = int((m.get("mask") or {}).get("size") or 0)
    o = np.zeros((T, H, dv))
    for i in range(T):
        js = [j for j in range(i + 1) if in_window(i, j, size)]
        lo = js[0]
        for a in range(H):
            s = (k[lo:i + 1, a] @ qn[i, a] + r[lo:i + 1] @ qr[i, a]) * float(m["scale"])
            o[i, a] = softmax(s) @ v[lo:i + 1, a]
    return o.reshape(T, H * dv) @ w[p + "o"].T


# -- feed-forward -----------------------------------------------------------------------------------------------------

def expert(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def mixture(mlp, w, p, x, tokens):
    """x [tokens, width]: the table gives every token id its experts, which count alike."""
    y = np.zeros_like(x)
    top = int(mlp["router"]["top"])
    for t, tok in enumerate(tokens):
        for e in w[p + "table"][tok]:
            y[t] += expert(w, f"{p}e{int(e)}.", x[t]) / top
    if mlp.get("shared"):
        y += expert(w, p + "shared.", x)
    return y


# -- the model --------------------------------------------------------------------------------------------------------

def layer(cfg, lc, w, i, x, tokens, first_values):
    """-> (the new stream, the first mixing layer's values from here on)."""
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg["postln_alpha"])
    p, m = f"l{i}.", lc["mixer"]
    if lc["type"] == "attention":
        mixes = bool(m.get("v_mix"))
        y, own = attention(m, w, p + "mix.", x, eps, first_values if mixes else None)
        if mixes and first_values is None:
            first_values = own
    elif lc["type"] == "latent_attention":
        y = latent_attention(m, w, p + "mix.", x, eps)
    else:
        raise ValueError(lc["type"])
    x = norm(alpha * x + y, w[p + "norm1"], eps)
    if lc.get("mlp") is not None:
        x = norm(alpha * x + mixture(lc["mlp"], w, p + "mlp.", x, tokens), w[p + "norm2"], eps)
    return x, first_values


def forward(cfg, w, tokens, keep_layers=False):
    """-> logits [tokens, vocab] (and the stream behind every layer)."""
    x = w["embed"][np.asarray(tokens)]
    kept, first = [], None
    for i, lc in enumerate(cfg["layers"]):
        x, first = layer(cfg, lc, w, i, x, tokens, first)
        kept.append(x.copy())
    logits = norm(x, w["final.norm"], float(cfg["norm"]["eps"])) @ w["head"].T
    cap = float(cfg.get("logit_softcap") or 0.0)
    if cap:
        logits = cap * np.tanh(logits / cap)
    return (logits, kept) if keep_layers else logits


def greedy(cfg, w, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(np.argmax(forward(cfg, w, ids)[-1])))
    return ids[len(prompt):]
