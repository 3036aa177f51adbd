"""A plain, slow implementation of the Sobezen decoder: the oracle of its tests.

Whole sequences, no cache, no batching, numpy only, float64 by default, one function per mechanism.  It shares no code with
the library (the model folder is read with the few lines of ``plain_llama.read_safetensors``, which is test code as well).

Notation: ``x`` is the residual stream [T, W]; a matrix is stored [out, in] and applied as ``x @ M.T``; T tokens at
positions 0 .. T-1.

The design, restated:

* the stream starts as the table's row times ``embedding.scale``;
* a layer is x += a * mixer(norm1(x)), then, where it has a feed-forward, x += b * ff(norm2(x)), with a learned vector
  each (a, b: a number per entry of the stream) and RMS norms;
* mixers: attention through a low-rank latent (a layer may read an earlier layer's latent rows instead of making its own),
  a gated delta rule whose decay has a number per key channel, or grouped-query attention whose values are its keys before
  the rotation;
* the feed-forward is gated: z * logistic(1.702 z) * (u + 1) with z bounded from above and u from both sides;
* a last RMS norm, a head, and one factor on all logits.
"""
from __future__ import annotations

import json
import math
import os

import numpy as np

from plain_llama import read_safetensors


def read_model(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ----------------------------------------------------------------------------- small pieces

def rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def logistic(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * logistic(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def softmax(z):
    e = np.exp(z - np.max(z, axis=-1, keepdims=True))
    return e / np.sum(e, axis=-1, keepdims=True)


def frequencies(rot):
    """-> (f [dims/2], amplitude).  Plain: base^(-2i/dims).  With ``scaling`` the slow pairs are divided by ``factor``, the
    fast ones kept, those between mixed linearly by index, and cos and sin grow by an amplitude."""
    d, base = rot["dims"], rot["base"]
    i = np.arange(d // 2, dtype=np.float64)
    f = float(base) ** (-2.0 * i / d) if d else np.zeros(0)
    s = rot.get("scaling")
    if s is None:
        return f, 1.0

    def index_of(turns):
        return d * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index_of(s["fast"])), 0), min(math.ceil(index_of(s["slow"])), d - 1)
    share = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / s["factor"] * share + f * (1.0 - share), 0.1 * math.log(s["factor"]) + 1.0


def rotate(v, rot):
    """Neighbouring entries (2i, 2i+1) of the first ``dims`` of the last axis turn by position * f_i.  v [T, ..., D]."""
    if not rot or not rot["dims"]:
        return v
    d = rot["dims"]
    f, amp = frequencies(rot)
    ang = np.arange(v.shape[0], dtype=np.float64)[:, None] * f[None, :]
    shape = (v.shape[0],) + (1,) * (v.ndim - 2) + (d // 2,)
    c, s = amp * np.cos(ang).reshape(shape), amp * np.sin(ang).reshape(shape)
    out = np.array(v, copy=True)
    a, b = v[..., 0:d:2], v[..., 1:d:2]
    out[..., 0:d:2] = a * c - b * s
    out[..., 1:d:2] = b * c + a * s
    return out


def short_conv(x, taps):
    """Per channel over time, x [T, C], taps [C, K]: the last column multiplies the current token; zeros before the start."""
    T, K = x.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((K - 1, x.shape[1]), dtype=x.dtype), x], axis=0)
    return sum(padded[j:j + T] * taps[None, :, j] for j in range(K))


# ----------------------------------------------------------------------------- mixers

def latent_rows(h, w, p, m, eps):
    """What a layer with a down-projection of its own keeps per token: (latent [T, C], rotated key part [T, R])."""
    down = h @ w[p + ".dkv"].T
    C = m["kv_rank"]
    return rms(down[:, :C], eps) * w[p + ".dkv.norm"], rotate(down[:, C:], m.get("rot"))


def latent_attention(h, w, p, m, eps, rows):
    """``rows``: the latent and the shared rotated key part that this layer reads (its own or an earlier layer's).  Every
    head's keys and values are written out; nothing is folded."""
    T = h.shape[0]
    H, D, R, Dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    c, k_rot = rows
    cq = rms(h @ w[p + ".dq"].T, eps) * w[p + ".dq.norm"]
    q = (cq @ w[p + ".uq"].T).reshape(T, H, D + R)
    q_plain, q_rot = q[..., :D], rotate(q[..., D:], m.get("rot"))
    k_plain = (c @ w[p + ".uk"].T).reshape(T, H, D)
    v = (c @ w[p + ".uv"].T).reshape(T, H, Dv)
    seen = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, Dv), dtype=h.dtype)
    for i in range(H):
        s = (q_plain[:, i] @ k_plain[:, i].T + q_rot[:, i] @ k_rot.T) * m["scale"]
        out[:, i] = softmax(np.where(seen, s, -np.inf)) @ v[:, i]
    return out.reshape(T, H * Dv) @ w[p + ".o"].T


def channel_decay(h, w, p, H, D):
    """g [T, H, D] in (0, 1): exp(-exp(A_log_h) * softplus(W_a2 W_a1 h + dt_bias))."""
    z = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".dt_bias"]
    return np.exp(-np.exp(w[p + ".A_log"])[None, :, None] * softplus(z).reshape(-1, H, D))


def delta_walk(q, k, v, beta, g):
    """The recurrence over tokens, all heads at once: q, k, g [T, H, D], v [T, H, Dv], beta [T, H] -> o [T, H, Dv].
    S <- g S (row by row);  u = beta (v - k S);  S <- S + k u;  o = q S."""
    T, H, D = k.shape
    S = np.zeros((H, D, v.shape[2]), dtype=v.dtype)
    o = np.zeros_like(v)
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hd,hdv->hv", k[t], S))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hd,hdv->hv", q[t], S)
    return o


def channel_delta(h, w, p, m, eps):
    T = h.shape[0]
    H, Hk, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def through(name, n, size):
        return silu(short_conv(h @ w[p + name].T, w[p + name + ".conv"])).reshape(T, n, size)
    q, k, v = through(".q", Hk, D), through(".k", Hk, D), through(".v", H, Dv)
    unit = lambda a: a / np.sqrt(np.sum(a * a, axis=-1, keepdims=True) + 1e-6)      # noqa: E731
    q, k = unit(q) * D ** -0.5, unit(k)
    of_head = np.arange(H) // (H // Hk)
    beta = logistic(h @ w[p + ".b"].T)
    o = delta_walk(q[:, of_head], k[:, of_head], v, beta, channel_decay(h, w, p, H, D))
    gate = logistic((h @ w[p + ".g1"].T) @ w[p + ".g2"].T).reshape(T, H, Dv)
    return (rms(o, eps) * w[p + ".norm"] * gate).reshape(T, H * Dv) @ w[p + ".o"].T


def grouped_attention(h, w, p, m):
    """Query head i reads key head i // (heads / kv_heads); the values are the keys as projected (bias in, not rotated)."""
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + ".q"].T + w[p + ".q.b"]).reshape(T, H, D)
    v = (h @ w[p + ".k"].T + w[p + ".k.b"]).reshape(T, G, D)
    q, k = rotate(q, m.get("rot")), rotate(v, m.get("rot"))
    seen = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, D), dtype=h.dtype)
    for i in range(H):
        j = i // (H // G)
        out[:, i] = softmax(np.where(seen, q[:, i] @ k[:, j].T * m["scale"], -np.inf)) @ v[:, j]
    return out.reshape(T, H * D) @ w[p + ".o"].T


# ----------------------------------------------------------------------------- feed-forward

def bounded_gate(z, u, limit):
    """z from above at ``limit``, u between -limit and limit;  z * logistic(1.702 z) * (u + 1)."""
    z, u = np.minimum(z, limit), np.clip(u, -limit, limit)
    return z * logistic(1.702 * z) * (u + 1.0)


def dense_ff(h, w, p, mlp):
    y = bounded_gate(h @ w[p + ".gate"].T + w[p + ".gate.b"], h @ w[p + ".up"].T + w[p + ".up.b"], mlp["limit"])
    return y @ w[p + ".down"].T + w[p + ".down.b"]


# ----------------------------------------------------------------------------- the model

def forward(cfg, w, tokens, dtype=np.float64, return_states=False):
    """Logits [T, vocab] of one whole sequence; with ``return_states`` also the stream after every layer."""
    w = {k: np.asarray(v, dtype=dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    states, rows = [], {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}", layer["mixer"]
        h = rms(x, eps) * w[p + ".norm1"]
        if layer["type"] == "latent_attention":
            j = m.get("kv_from")
            if j is None:
                rows[i] = latent_rows(h, w, p + ".mix", m, eps)
            y = latent_attention(h, w, p + ".mix", m, eps, rows[i if j is None else j])
        elif layer["type"] == "channel_delta":
            y = channel_delta(h, w, p + ".mix", m, eps)
        elif layer["type"] == "attention":
            y = grouped_attention(h, w, p + ".mix", m)
        else:
            raise ValueError(layer["type"])
        x = x + y * w[p + ".ls1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms(x, eps) * w[p + ".norm2"]
            x = x + dense_ff(h, w, p + ".mlp", mlp) * w[p + ".ls2"]
        states.append(x.copy())
    logits = (rms(x, eps) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]
    return (logits, states) if return_states else logits


def generate_greedy(cfg, w, prompt, max_new, dtype=np.float64):
    toks, out = list(prompt), []
    for _ in range(max_new):
        nxt = int(np.argmax(forward(cfg, w, toks, dtype)[-1]))
        out.append(nxt)
        toks.append(nxt)
    return out
