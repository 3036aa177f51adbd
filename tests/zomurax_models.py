"""Small Zomurax configurations and weights for the tests: sizes unlike one another (and unlike any model the library
ships numbers for), and weights large enough that every mechanism matters: sharp attention, distance biases from nearly
none to steep, sinks that take a good part of a softmax, tables that send neighbouring ids to different experts."""
import json
import os

import numpy as np


def att(heads, kv_heads, dim, vdim, scale=None, mix=True, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": float(scale if scale is not None else 1.8 * dim ** -0.5)}
    if mix is not None:
        m["v_mix"] = mix
    if temp is not None:
        m["q_temp"] = {"coef": float(temp[0]), "every": temp[1]}
    return "attention", m


def lat(heads, dim, rot_dim, vdim, rank, window=None, base=10000.0, scale=None, dims=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
         "scale": float(scale if scale is not None else 1.0 * (dim + rot_dim) ** -0.5)}
    if rot_dim:
        m["rot"] = {"base": float(base), "dims": rot_dim if dims is None else dims}
    if window is not None:
        m["mask"] = {"size": window}
    return "latent_attention", m


def moe(ff, experts, top, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, eps=1e-5, alpha=1.5, cap=12.0):
    return {"architecture": "Zomurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": float(alpha),
            "logit_softcap": float(cap), "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


# one mechanism at a time
ATT = config(40, 83, [(att(6, 2, 12, 20, temp=(0.5, 7)), None), (att(5, 5, 16, 8, mix=False), None)], alpha=0.8)
MIX = config(48, 71, [(att(4, 4, 8, 6, mix=False, temp=(0.3, 50)), None), (att(6, 3, 10, 8, temp=(0.2, 1)), None), (lat(3, 8, 4, 12, 20, 9), None),
                      (att(2, 2, 24, 12), None), (att(4, 1, 16, 24, temp=(-0.1, 33)), None)], alpha=2.0)      # 24 values a token in every layer that mixes
LAT = config(44, 97, [(lat(5, 12, 8, 6, 28, 17, base=300.0), None), (lat(2, 16, 6, 10, 36, 64, dims=4), None)], alpha=1.0)
LAT_BARE = config(36, 61, [(lat(3, 8, 0, 8, 16), None), (lat(4, 6, 2, 9, 12, 1), None)], alpha=1.2)     # no rotated part and no window; a window of one
EXPERTS = config(40, 90, [(lat(2, 8, 4, 8, 16, 30), moe(16, 5, 3, shared=24)), (att(2, 1, 8, 8), moe(12, 4, 1)),
                          (lat(1, 8, 2, 8, 8, 12), moe(8, 3, 3, shared=8))], cap=5.0)                   # one choice without a shared expert; all experts chosen
# layers unlike each other: windows as long as a page, a little longer, longer than two, dividing no page
MIXED = config(56, 120, [(lat(4, 12, 4, 8, 24, 70, base=1000.0), moe(24, 6, 2, shared=16)), (att(4, 2, 12, 8, temp=(0.4, 40)), None),
                         (att(8, 2, 16, 8), moe(16, 3, 2)), (lat(6, 8, 8, 4, 40, 65), moe(8, 8, 3, shared=40)),
                         (lat(3, 20, 2, 12, 12, 150), None), (att(1, 1, 20, 16, scale=1.1, temp=(0.7, 200)), moe(16, 4, 2, shared=8))],
               eps=1e-4, alpha=2.5, cap=20.0)
# sizes of the kind the fast kernels take (multiples of 16 and 64), several layers
WIDE = config(128, 300, [(att(4, 2, 64, 64, temp=(0.3, 60)), moe(64, 8, 2, shared=128)), (lat(4, 64, 32, 64, 128, 100, base=50000.0), moe(128, 4, 2, shared=64)),
                         (att(8, 2, 32, 64), None), (lat(16, 32, 64, 16, 64, 129), moe(64, 16, 4)), (att(2, 1, 128, 128), moe(64, 6, 3, shared=64))], cap=15.0)
# sizes that fit no fast kernel: rows of odd byte counts, head counts that divide nothing
ODD = config(36, 77, [(att(5, 5, 6, 9, temp=(0.25, 11)), moe(10, 3, 2, shared=7)), (lat(3, 6, 6, 7, 11, 13, base=50.0), moe(22, 5, 2)),
                      (att(10, 5, 7, 9), None)], eps=1e-6, alpha=1.1)
# a width and sizes that are no multiples of four: nothing is aligned to 16 bytes
UNALIGNED = config(50, 101, [(lat(3, 7, 2, 9, 13, 20), moe(11, 3, 2, shared=13)), (att(2, 1, 10, 6, temp=(0.9, 5)), moe(9, 2, 1)), (att(3, 3, 5, 2), None)],
                   alpha=0.7)
CONFIGS = {"unaligned": UNALIGNED, "att": ATT, "mix": MIX, "lat": LAT, "lat_bare": LAT_BARE, "experts": EXPERTS, "mixed": MIXED, "wide": WIDE, "odd": ODD}


def make_weights(cfg, seed):
    """name -> float32 array (int32 for the tables)."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def mat(name, out, inp, gain=1.0):
        w[name] = (rng.standard_normal((out, inp)) * gain / np.sqrt(inp)).astype(np.float32)

    def one(name, mean, std):
        w[name] = np.float32(mean + std * rng.standard_normal())

    w["embed"] = rng.standard_normal((V, W)).astype(np.float32)
    mat("head", V, W, 2.0)
    one("final.norm", 1.1, 0.2)
    mixing = False
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        one(p + "norm1", 1.0, 0.2)
        if layer["type"] == "attention":
            H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            mat(p + "mix.q", H * D, W)
            mat(p + "mix.k", G * D, W)
            mat(p + "mix.v", G * Dv, W, 2.0)
            mat(p + "mix.o", W, H * Dv, 1.5)
            r1 = rng.uniform(0.3, 2.0, H)
            r1[rng.integers(0, H)] = 0.03                  # one head looks far back
            w[p + "mix.r1"] = r1.astype(np.float32)
            w[p + "mix.r2"] = rng.uniform(0.05, 0.6, H).astype(np.float32)
            w[p + "mix.sink"] = rng.uniform(0.0, 4.0, H).astype(np.float32)
            if m.get("v_mix") and mixing:
                w[p + "mix.vmix"] = np.float32(rng.uniform(0.2, 0.8))
            mixing = mixing or bool(m.get("v_mix"))
        else:
            H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            mat(p + "mix.q", H * (D + R), W, 1.5)
            mat(p + "mix.dkv", C + R, W, 1.5)
            w[p + "mix.dkv.norm"] = (1.0 + 0.2 * rng.standard_normal(C)).astype(np.float32)
            mat(p + "mix.uk", H * D, C)
            mat(p + "mix.uv", H * Dv, C, 2.0)
            mat(p + "mix.o", W, H * Dv, 1.5)
        mlp = layer["mlp"]
        if mlp is not None:
            one(p + "norm2", 1.0, 0.2)
            F, E, top = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"]
            for e in range(E):
                for n in ("gate", "up"):
                    mat(f"{p}mlp.e{e}.{n}", F, W)
                mat(f"{p}mlp.e{e}.down", W, F, 1.5)
            w[p + "mlp.table"] = np.argsort(rng.random((V, E)), axis=1)[:, :top].astype(np.int32)
            if mlp.get("shared"):
                S = mlp["shared"]["ff"]
                for n in ("gate", "up"):
                    mat(f"{p}mlp.shared.{n}", S, W)
                mat(p + "mlp.shared.down", W, S)
    return w


def write_model(folder, cfg, weights, storage="F32"):
    """config.json and model.safetensors; ``storage`` F32 or BF16 for all but the tables.  Returns the weights as the file
    holds them (float64; tables as they are)."""
    import torch
    from llmi_b200.weights.safetensors_io import write_safetensors
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    dt = {"F32": torch.float32, "BF16": torch.bfloat16}[storage]
    tensors = {}
    for k, v in weights.items():
        t = torch.from_numpy(np.array(v))
        tensors[k] = t if t.dtype == torch.int32 else t.to(dt)
    write_safetensors(os.path.join(folder, "model.safetensors"), tensors, metadata={"format": "pt"})
    return {k: t.numpy() if t.dtype == torch.int32 else t.float().numpy().astype(np.float64) for k, t in tensors.items()}
