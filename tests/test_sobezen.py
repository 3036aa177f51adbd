"""The Sobezen design on the CPU: its configuration and what it refuses, the recipe and its tensor table, random folders,
and the plain implementation's own mechanisms."""
import copy
import math

import numpy as np
import pytest

import plain_sobezen as G
import sobezen_models as M


def test_configuration_reads_every_size_and_refuses_what_is_wrong():
    from llmi_b200.config import ConfigError
    from llmi_b200.config.registry import parse_config
    arch, c = parse_config(M.MIXED)
    assert arch.name == "Sobezen" and (c.width, c.vocab, c.norm_eps, c.embedding_scale, c.logit_scale) == (56, 120, 1e-4, 3.0, 0.7)
    assert [layer.type for layer in c.layers] == [layer["type"] for layer in M.MIXED["layers"]]
    d, t, a, s = c.layers[4].mixer, c.layers[1].mixer, c.layers[5].mixer, c.layers[3].mixer
    assert (d.heads, d.kv_heads, d.dim, d.vdim, d.conv) == (6, 3, 12, 8, 4)
    assert (t.heads, t.dim, t.rot_dim, t.vdim, t.kv_rank, t.q_rank, t.kv_from) == (6, 10, 8, 12, 36, 18, None)
    assert (t.rot.base, t.rot.dims, t.rot.scaling.factor, t.rot.scaling.original, t.rot.scaling.fast, t.rot.scaling.slow) == (2000.0, 8, 8.0, 64, 16.0, 1.0)
    assert (s.kv_from, s.heads, s.q_rank) == (1, 2, 30) and (a.heads, a.kv_heads, a.dim, a.rot.base, a.rot.dims, a.rot.scaling) == (8, 2, 16, 700.0, 8, None)
    assert c.layers[0].mlp.ff == 40 and c.layers[0].mlp.limit == 1.0 and c.layers[2].mlp is None
    for path, value in ((("width",), None), (("embedding",), {}), (("logit_scale",), None), (("norm",), {}), (("layers", 0, "type"), "delta"), (("layers",), []),
                        (("layers", 0, "mixer", "heads"), 0), (("layers", 0, "mixer", "kv_heads"), 3), (("layers", 0, "mixer", "conv"), 0),
                        (("layers", 0, "mixer", "conv"), 17), (("layers", 0, "mixer", "vdim"), None), (("layers", 1, "mixer", "kv_rank"), None),
                        (("layers", 1, "mixer", "q_rank"), 0), (("layers", 1, "mixer", "scale"), 0), (("layers", 1, "mixer", "rot", "dims"), 7),
                        (("layers", 1, "mixer", "rot", "dims"), 10), (("layers", 1, "mixer", "rot", "base"), 1.0),
                        (("layers", 1, "mixer", "rot", "scaling", "factor"), None), (("layers", 2, "mixer", "vdim"), 8), (("layers", 2, "mixer", "kv_heads"), 3),
                        (("layers", 3, "mixer", "kv_from"), 0), (("layers", 3, "mixer", "kv_from"), 3), (("layers", 3, "mixer", "kv_from"), -1),
                        (("layers", 3, "mixer", "kv_rank"), 20), (("layers", 3, "mixer", "rot", "base"), 100.0), (("layers", 0, "mlp", "kind"), "moe"),
                        (("layers", 0, "mlp", "limit"), None), (("layers", 0, "mlp", "ff"), 0), (("layers", 0, "mlp"), 3)):
        bad = copy.deepcopy(M.MIXED)
        node = bad
        for key in path[:-1]:
            node = node[key]
        if value is None:
            del node[path[-1]]
        else:
            node[path[-1]] = value
        with pytest.raises(ConfigError):
            parse_config(bad)
    chain = copy.deepcopy(M.SHARED)
    chain["layers"][5]["mixer"]["kv_from"] = 3                        # a layer whose own rows are another layer's
    with pytest.raises(ConfigError):
        parse_config(chain)


def test_recipe_and_tensor_table():
    from llmi_b200.config.registry import parse_config
    from llmi_b200.parts.build import expected_tensors
    from llmi_b200.parts.registry import FreeDim
    for name, cfg in M.CONFIGS.items():
        arch, c = parse_config(cfg)
        spec = arch.model_spec(c)
        assert [e.layer for e in spec.schedule] == list(range(len(cfg["layers"])))
        assert [e.cache_of for e in spec.schedule] == [layer["mixer"].get("kv_from") for layer in cfg["layers"]]
        decl, made = expected_tensors(spec), M.make_weights(cfg, 1)
        assert set(decl) == set(made), (name, set(decl) ^ set(made))
        for n, d in decl.items():
            assert len(d.shape) == np.ndim(made[n]) and all(isinstance(a, FreeDim) or a == b for a, b in zip(d.shape, np.shape(made[n]))), (name, n)
    assert arch.tolerated_extra_tensors("l3.norm2") and arch.tolerated_extra_tensors("l0.ls2")
    assert not arch.tolerated_extra_tensors("l0.ls1") and not arch.tolerated_extra_tensors("l0.mix.v")


def test_a_random_folder_has_the_recipes_tensors(tmp_path):
    import torch
    from llmi_b200.config.registry import parse_config
    from llmi_b200.parts.build import expected_tensors
    from llmi_b200.parts.registry import resolved_shape
    from llmi_b200.weights.random_weights import write_random_model
    from llmi_b200.weights.safetensors_io import SafetensorsFile
    cfg = M.CONFIGS["mixed"]
    write_random_model(str(tmp_path), cfg, seed=3, dtype=torch.bfloat16)
    arch, c = parse_config(cfg)
    decl = expected_tensors(arch.model_spec(c))
    f = SafetensorsFile(str(tmp_path / "model.safetensors"))
    try:
        assert set(f.names()) == set(decl)
        for n, d in decl.items():
            assert tuple(f.tensor(n).shape) == resolved_shape(d.shape), n
    finally:
        f.close()


# ---------------------------------------------------------------------------------- the oracle's own mechanisms

def test_stretched_frequencies_and_rotation():
    rot = {"base": 10000.0, "dims": 8}
    f, amp = G.frequencies(rot)
    assert np.allclose(f, [1.0, 0.1, 0.01, 0.001]) and amp == 1.0
    stretched = dict(rot, scaling={"factor": 4.0, "original": 2 * math.pi * 1000, "fast": 1000.0, "slow": 10.0})
    f2, amp2 = G.frequencies(stretched)                      # pair indices 0 (1000 turns) and 2 (10 turns): kept, half way, divided
    assert np.allclose(f2, [1.0, 0.1 * (0.5 + 0.125), 0.01 / 4, 0.001 / 4]) and np.isclose(amp2, 1 + 0.1 * math.log(4.0))
    v = np.random.default_rng(0).standard_normal((5, 2, 10))
    y = G.rotate(v, stretched)
    assert np.allclose(y[..., 8:], v[..., 8:]) and np.allclose(y[0, :, :8], amp2 * v[0, :, :8])
    assert np.allclose(np.hypot(y[..., 2], y[..., 3]), amp2 * np.hypot(v[..., 2], v[..., 3]))
    assert np.allclose(y[3, 0, 0], amp2 * (v[3, 0, 0] * math.cos(3) - v[3, 0, 1] * math.sin(3)))
    assert np.array_equal(G.rotate(v, {"base": 10.0, "dims": 0}), v)


def test_the_walk_writes_before_it_reads_and_decays_rows():
    """One head, by hand: a first token writes beta v kᵀ; a second one sees it through its own rows' decay."""
    k, q = np.zeros((2, 1, 3)), np.zeros((2, 1, 3))
    k[0, 0, 0] = k[1, 0, 1] = 1.0
    q[0, 0] = [2.0, 0.0, 0.0]
    q[1, 0] = [1.0, 1.0, 0.0]
    v = np.array([[[3.0, 1.0]], [[0.0, 5.0]]])
    g = np.array([[[0.9, 0.9, 0.9]], [[0.5, 0.1, 0.7]]])
    o = G.delta_walk(q, k, v, np.array([[0.5], [1.0]]), g)
    assert np.allclose(o[0, 0], [3.0, 1.0])                  # 2 * (0.5 v): the read-out sees the token's own write
    assert np.allclose(o[1, 0], 0.5 * np.array([1.5, 0.5]) + [0.0, 5.0])
    again = G.delta_walk(q[:1].repeat(2, 0), k[:1].repeat(2, 0), v[:1].repeat(2, 0), np.ones((2, 1)), np.ones((2, 1, 3)))
    assert np.allclose(again[1], again[0])                   # a full write of what is there changes nothing


def test_bounded_gate_and_convolution():
    z, u = np.array([-3.0, 0.5, 9.0]), np.array([-9.0, 0.2, 9.0])
    y = G.bounded_gate(z, u, 2.0)
    assert np.isclose(y[2], 2.0 / (1 + math.exp(-1.702 * 2)) * 3.0) and np.isclose(y[1], 0.5 / (1 + math.exp(-0.851)) * 1.2)
    assert np.isclose(y[0], -3.0 / (1 + math.exp(1.702 * 3)) * -1.0)             # no bound from below on the gate
    x = np.array([[1.0], [2.0], [3.0]])
    assert np.allclose(G.short_conv(x, np.array([[10.0, 1.0]]))[:, 0], [1.0, 12.0, 23.0])


def test_a_sharing_layer_reads_the_other_layers_rows_and_not_its_own_input():
    cfg = M.CONFIGS["shared"]
    w = M.make_weights(cfg, 3)
    toks = [1, 5, 9, 44, 2]
    base = G.forward(cfg, w, toks)
    m = copy.deepcopy(cfg)
    del m["layers"][3]["mixer"]["kv_from"]
    w2 = dict(w)
    for n in ("dkv", "dkv.norm"):
        w2["l3.mix." + n] = w["l0.mix." + n]
    assert not np.allclose(base, G.forward(m, w2, toks))


def test_latent_attention_with_folded_expansions():
    """Uk_hᵀ q . c is q . Uk_h c, and the values' expansion can follow the weighted sum."""
    cfg = M.CONFIGS["lat"]
    m, eps = cfg["layers"][0]["mixer"], 1e-5
    w = {k: np.asarray(v, dtype=np.float64) for k, v in M.make_weights(cfg, 2).items()}
    x = np.random.default_rng(0).standard_normal((30, cfg["width"]))
    c, kr = G.latent_rows(x, w, "l0.mix", m, eps)
    y = G.latent_attention(x, w, "l0.mix", m, eps, (c, kr))
    H, D, R, Dv, C = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    q = ((G.rms(x @ w["l0.mix.dq"].T, eps) * w["l0.mix.dq.norm"]) @ w["l0.mix.uq"].T).reshape(30, H, D + R)
    qr = G.rotate(q[..., D:], m["rot"])
    uk, uv = w["l0.mix.uk"].reshape(H, D, C), w["l0.mix.uv"].reshape(H, Dv, C)
    o = np.zeros((30, H, Dv))
    for t in range(30):
        for a in range(H):
            s = (c[:t + 1] @ (uk[a].T @ q[t, a, :D]) + kr[:t + 1] @ qr[t, a]) * m["scale"]
            o[t, a] = uv[a] @ (G.softmax(s) @ c[:t + 1])
    assert np.allclose(y, o.reshape(30, -1) @ w["l0.mix.o"].T)
