"""Small Sobezen configurations and weights for the tests: sizes unlike one another, and weights large enough that every
mechanism matters: sharp attention, biases that move keys and values, gates driven past their bounds, layer factors far
from one, decays from nearly one to fast."""
import json
import os

import numpy as np


def lat(heads, dim, rot_dim, vdim, kv_rank, q_rank, base=10000.0, scaling=None, scale=None, kv_from=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
         "scale": float(scale if scale is not None else 1.3 * (dim + rot_dim) ** -0.5), "rot": {"base": float(base), "dims": rot_dim}}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "latent_attention", m


def delta(heads, kv_heads, dim, vdim, conv):
    return "channel_delta", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def att(heads, kv_heads, dim, rot=None, base=10000.0, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": float(scale if scale is not None else 1.5 * dim ** -0.5),
                         "rot": {"base": float(base), "dims": dim if rot is None else rot}}


def ff(inner, limit):
    return {"kind": "dense", "ff": inner, "limit": float(limit)}


def config(width, vocab, layers, eps=1e-5, scale=3.0, logit_scale=0.7):
    return {"architecture": "Sobezen", "vocab": vocab, "width": width, "embedding": {"scale": float(scale)}, "norm": {"eps": eps},
            "logit_scale": float(logit_scale), "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


# one mechanism at a time
LAT = config(44, 97, [(lat(3, 12, 6, 10, 20, 14, scaling=(4.0, 40, 8.0, 1.0), base=300.0), None), (lat(5, 8, 4, 6, 28, 9), None)], scale=1.0)
# rows shared: two layers on the first one's rows, one on the third's, with layers of other kinds between them
SHARED = config(40, 83, [(lat(2, 8, 8, 12, 16, 10), ff(24, 1.5)), (att(2, 1, 8), None), (lat(4, 10, 4, 6, 24, 12, base=500.0), None),
                         (lat(3, 14, 8, 5, 16, 22, kv_from=0), None), (lat(1, 6, 4, 9, 24, 7, base=500.0, kv_from=2), ff(16, 3.0)),
                         (lat(5, 4, 8, 8, 16, 6, scale=0.6, kv_from=0), None)], logit_scale=1.3)
DELTA = config(40, 71, [(delta(4, 2, 24, 20, 4), None), (delta(3, 1, 20, 12, 2), None)])
DELTA_ONE_TAP = config(32, 64, [(delta(2, 2, 8, 36, 1), None), (delta(1, 1, 10, 7, 5), ff(20, 2.0))])     # (10, 7: no 16-byte columns)
ATT = config(36, 90, [(att(6, 2, 10, rot=4), None), (att(3, 3, 14, rot=0), None), (att(4, 1, 8, base=50.0), None)], eps=1e-4)
GATE = config(48, 61, [(att(1, 1, 8), ff(72, 0.4)), (att(2, 2, 6, rot=2), ff(10, 5.0))], scale=0.8)
# layers unlike each other, one of each kind without a feed-forward
MIXED = config(56, 120, [(delta(4, 4, 16, 24, 3), ff(40, 1.0)), (lat(6, 10, 8, 12, 36, 18, scaling=(8.0, 64, 16.0, 1.0), base=2000.0), ff(64, 2.5)),
                         (att(4, 2, 12), None), (lat(2, 16, 8, 6, 36, 30, scaling=(8.0, 64, 16.0, 1.0), base=2000.0, kv_from=1), None),
                         (delta(6, 3, 12, 8, 4), None), (att(8, 2, 16, rot=8, base=700.0), ff(24, 0.8))], eps=1e-4)
# sizes of the kind the fast kernels take (multiples of 16 and 64), several layers
WIDE = config(128, 300, [(lat(8, 32, 32, 64, 64, 64, scaling=(16.0, 100, 8.0, 2.0), base=50000.0), ff(192, 1.5)), (delta(4, 2, 64, 64, 4), ff(128, 2.0)),
                         (att(4, 2, 64), None), (lat(2, 64, 32, 32, 64, 128, scaling=(16.0, 100, 8.0, 2.0), base=50000.0, kv_from=0), ff(64, 1.0)),
                         (delta(2, 2, 128, 96, 2), None), (att(6, 3, 80, rot=32), ff(64, 4.0)), (delta(3, 3, 32, 48, 3), None), (att(2, 1, 128), None)],
              scale=2.0)
# sizes that fit no fast kernel: rows of odd byte counts, head counts that divide nothing
ODD = config(50, 77, [(delta(3, 3, 5, 9, 2), ff(11, 1.2)), (lat(3, 7, 2, 9, 13, 11), ff(22, 0.9)), (att(5, 5, 6, rot=2), None),
                      (lat(2, 3, 2, 4, 13, 5, kv_from=1), None)], eps=1e-6, logit_scale=2.0)
ONE = config(16, 20, [(lat(1, 4, 2, 4, 8, 4), None)], logit_scale=1.0, scale=1.0)
CONFIGS = {"lat": LAT, "shared": SHARED, "delta": DELTA, "delta_one_tap": DELTA_ONE_TAP, "att": ATT, "gate": GATE, "mixed": MIXED, "wide": WIDE,
           "odd": ODD, "one": ONE}


def make_weights(cfg, seed, keep_state=False):
    """name -> float32 array.  ``keep_state``: decays next to one, so that a state that is lost or cut anywhere changes
    everything after it."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = (rng.standard_normal((out, inp)) * gain / np.sqrt(inp)).astype(np.float32)

    def near_one(name, n, std=0.2):
        w[name] = (1.0 + std * rng.standard_normal(n)).astype(np.float32)

    def vec(name, n, std):
        w[name] = (std * rng.standard_normal(n)).astype(np.float32)

    w["embed"] = (rng.standard_normal((V, W)) / cfg["embedding"]["scale"]).astype(np.float32)
    mat("head", V, W, 2.0)
    near_one("final.norm", W)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        near_one(p + "norm1", W)
        near_one(p + "ls1", W, 0.5)
        if layer["type"] == "latent_attention":
            H, D, R, Dv, C, Q = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            mat(p + "mix.dq", Q, W)
            near_one(p + "mix.dq.norm", Q)
            mat(p + "mix.uq", H * (D + R), Q, 2.0)
            if "kv_from" not in m:
                mat(p + "mix.dkv", C + R, W, 1.5)
                near_one(p + "mix.dkv.norm", C)
            mat(p + "mix.uk", H * D, C, 1.5)
            mat(p + "mix.uv", H * Dv, C)
            mat(p + "mix.o", W, H * Dv, 1.5)
        elif layer["type"] == "channel_delta":
            H, Hk, D, Dv, K = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            ra, rg = 3 + i, 6 + 2 * i                      # inner sizes of the low-rank paths: of the file's choosing
            for n, rows in (("q", Hk * D), ("k", Hk * D), ("v", H * Dv)):
                mat(p + "mix." + n, rows, W, 1.5)
                w[p + f"mix.{n}.conv"] = (rng.standard_normal((rows, K)) / np.sqrt(K)).astype(np.float32)
            mat(p + "mix.b", H, W, 2.0)
            mat(p + "mix.a1", ra, W)
            mat(p + "mix.a2", H * D, ra, 2.0)
            mat(p + "mix.g1", rg, W)
            mat(p + "mix.g2", H * Dv, rg, 2.0)
            vec(p + "mix.dt_bias", H * D, 1.0)
            w[p + "mix.A_log"] = (np.full(H, -9.0) if keep_state else np.log(rng.uniform(0.02, 1.5, H))).astype(np.float32)
            near_one(p + "mix.norm", Dv)
            mat(p + "mix.o", W, H * Dv, 1.5)
        else:
            H, G, D = m["heads"], m["kv_heads"], m["dim"]
            mat(p + "mix.q", H * D, W)
            vec(p + "mix.q.b", H * D, 0.5)
            mat(p + "mix.k", G * D, W)
            vec(p + "mix.k.b", G * D, 0.5)
            mat(p + "mix.o", W, H * D, 1.5)
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            near_one(p + "norm2", W)
            near_one(p + "ls2", W, 0.5)
            for n in ("gate", "up"):
                mat(p + "mlp." + n, F, W, 1.5)
                vec(p + f"mlp.{n}.b", F, 0.5)
            mat(p + "mlp.down", W, F)
            vec(p + "mlp.down.b", W, 0.3)
    return w


def write_model(folder, cfg, weights, storage="F32"):
    """config.json and model.safetensors; ``storage`` F32 or BF16.  Returns the weights as the file holds them (float64)."""
    import torch
    from llmi_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    dt = {"F32": torch.float32, "BF16": torch.bfloat16}[storage]
    tensors = {k: torch.from_numpy(np.array(v, dtype=np.float32)).to(dt) for k, v in weights.items()}
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})
    return {k: t.float().numpy().astype(np.float64) for k, t in tensors.items()}
