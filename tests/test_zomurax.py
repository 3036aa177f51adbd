"""The Zomurax design on the CPU: its configuration and what it refuses, the recipe and its tensor table, random folders,
and the plain implementation's own mechanisms."""
import copy
import math

import numpy as np
import pytest

import plain_zomurax as G
import zomurax_models as M


def test_configuration_reads_every_size_and_refuses_what_is_wrong():
    from llmi_b200.config import ConfigError
    from llmi_b200.config.registry import parse_config
    arch, c = parse_config(M.MIXED)
    assert arch.name == "Zomurax" and c.width == 56 and c.vocab == 120 and c.norm_eps == 1e-4 and len(c.layers) == 6
    assert c.alpha == 2.5 and c.logit_softcap == 20.0
    a, t = c.layers[1].mixer, c.layers[0].mixer
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.temp_coef, a.temp_every, a.v_mix) == (4, 2, 12, 8, 0.4, 40, True)
    assert (t.heads, t.dim, t.rot_dim, t.vdim, t.kv_rank, t.rot_base, t.rot_dims, t.window) == (4, 12, 4, 8, 24, 1000.0, 4, 70)
    f = c.layers[0].mlp
    assert (f.ff, f.experts, f.top, f.shared_ff) == (24, 6, 2, 16) and c.layers[1].mlp is None and c.layers[2].mlp.shared_ff == 0
    assert parse_config(M.ATT)[1].layers[1].mixer.temp_every == 0 and not parse_config(M.ATT)[1].layers[1].mixer.v_mix
    bare = parse_config(M.LAT_BARE)[1].layers[0].mixer
    assert (bare.rot_dim, bare.rot_dims, bare.window) == (0, 0, 0)
    other = copy.deepcopy(M.MIXED)
    other["layers"][1]["mixer"]["q_temp"]["every"] = 40.0          # a count without a fraction
    del other["layers"][2]["mixer"]["v_mix"], other["logit_softcap"]
    o = parse_config(other)[1]
    assert o.layers[1].mixer.temp_every == 40 and not o.layers[2].mixer.v_mix and o.logit_softcap == 0.0
    for path, value in ((("width",), None), (("postln_alpha",), None), (("norm",), {}), (("layers", 0, "type"), "delta"), (("logit_softcap",), -1.0),
                        (("layers", 1, "mixer", "heads"), 0), (("layers", 1, "mixer", "kv_heads"), 3), (("layers", 1, "mixer", "vdim"), None),
                        (("layers", 1, "mixer", "vdim"), 12), (("layers", 1, "mixer", "v_mix"), 1), (("layers", 1, "mixer", "scale"), 0),
                        (("layers", 1, "mixer", "q_temp", "every"), 0), (("layers", 1, "mixer", "q_temp", "every"), 1.5),
                        (("layers", 1, "mixer", "q_temp", "coef"), None), (("layers", 0, "mixer", "rot", "dims"), 6),
                        (("layers", 0, "mixer", "rot", "dims"), 3), (("layers", 0, "mixer", "rot", "base"), None),
                        (("layers", 0, "mixer", "mask", "size"), 0), (("layers", 0, "mixer", "kv_rank"), None),
                        (("layers", 0, "mlp", "router", "top"), 7), (("layers", 0, "mlp", "kind"), "dense"),
                        (("layers", 0, "mlp", "expert"), None), (("layers", 0, "mlp", "shared", "ff"), 0)):
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


def test_recipe_and_tensor_table():
    from llmi_b200.config.registry import parse_config
    from llmi_b200.parts.build import expected_tensors
    for name, cfg in M.CONFIGS.items():
        arch, c = parse_config(cfg)
        spec = arch.model_spec(c)
        assert [e.layer for e in spec.schedule] == list(range(len(cfg["layers"])))
        assert all(ls.block == "postnorm" and ls.block_params == {"alpha": cfg["postln_alpha"]} for ls in spec.layers)
        decl, made = expected_tensors(spec), M.make_weights(cfg, 1)
        assert set(decl) == set(made), (name, set(decl) ^ set(made))
        for n, d in decl.items():
            assert tuple(d.shape) == np.shape(made[n]) and (d.role == "int_table") == (np.asarray(made[n]).dtype == np.int32), (name, n)
    mixes = [ls.mixer.params.get("value_mix") for ls in arch.model_spec(parse_config(M.MIX)[1]).layers]
    assert mixes == [None, "first", None, "later", "later"]


def test_unused_numbers_of_a_file_are_not_refused():
    from llmi_b200.config.registry import parse_config
    arch, _ = parse_config(M.MIX)
    assert arch.tolerated_extra_tensors("l0.mix.vmix") and arch.tolerated_extra_tensors("l3.norm2")
    assert not arch.tolerated_extra_tensors("l0.mix.vmix2") and not arch.tolerated_extra_tensors("l0.mix.q.b")


def test_a_random_folder_has_the_recipes_tensors_and_sound_tables(tmp_path):
    from llmi_b200.config.registry import parse_config
    from llmi_b200.parts.build import expected_tensors
    from llmi_b200.weights.random_weights import write_random_model
    from llmi_b200.weights.safetensors_io import SafetensorsFile
    import torch
    cfg = M.CONFIGS["mixed"]
    write_random_model(str(tmp_path), cfg, seed=3, dtype=torch.bfloat16)
    arch, c = parse_config(cfg)
    decl = expected_tensors(arch.model_spec(c))
    f = SafetensorsFile(str(tmp_path / "model.safetensors"))
    try:
        assert set(f.names()) == set(decl)
        for n, d in decl.items():
            t = f.tensor(n).clone()                                              # (the file's own memory goes with it)
            assert tuple(t.shape) == tuple(d.shape), n
            if d.role == "int_table":
                assert t.dtype == torch.int32 and int(t.min()) >= 0 and int(t.max()) == d.high - 1
                assert all(len(set(r)) == len(r) for r in t.tolist())            # the entries of a row differ
            else:
                assert t.dtype == torch.bfloat16
    finally:
        f.close()


# ---------------------------------------------------------------------------------- the oracle's own mechanisms

def test_softmax_with_a_sink_distance_temperature_and_window():
    z = np.array([0.5, -1.0, 2.0])
    p = G.softmax(z, 1.0)
    total = np.exp(z).sum() + math.e
    assert np.allclose(p, np.exp(z) / total) and p.sum() < 1 and np.allclose(G.softmax(z).sum(), 1)
    assert np.allclose(G.softmax(z, 200.0), 0) and np.allclose(G.softmax(z, -200.0), G.softmax(z))
    assert G.distance_bias(0, 3.0, 0.5) == 0 and np.isclose(G.distance_bias(2, 3.0, 0.5), 3 * math.log(2))
    assert np.allclose(np.exp(-G.distance_bias(np.arange(4.0), 2.0, 1.0)), [1, 1 / 4, 1 / 9, 1 / 16])
    assert G.temperature(0, 0.5, 4) == 1 and G.temperature(2, 0.5, 4) == 1
    assert np.isclose(G.temperature(3, 0.5, 4), 1 + 0.5 * math.log(2)) and np.isclose(G.temperature(7, 0.5, 4), 1 + 0.5 * math.log(3))
    assert [j for j in range(12) if G.in_window(11, j, 3)] == [9, 10, 11] and [j for j in range(4) if G.in_window(2, j, 9)] == [0, 1, 2]
    assert [j for j in range(6) if G.in_window(4, j, 0)] == [0, 1, 2, 3, 4] and [j for j in range(6) if G.in_window(4, j, 1)] == [4]
    x = np.arange(1.0, 13.0).reshape(2, 6)
    y = G.rotate_half(x, 3, 100.0, 4)
    assert np.allclose(y[:, 4:], x[:, 4:]) and np.allclose(np.hypot(y[:, 0], y[:, 2]), np.hypot(x[:, 0], x[:, 2]))
    assert np.allclose(y[0, 0], x[0, 0] * np.cos(3.0) - x[0, 2] * np.sin(3.0)) and np.allclose(y[0, 1], x[0, 1] * np.cos(0.3) - x[0, 3] * np.sin(0.3))


def test_a_latent_layer_is_attention_with_folded_matrices():
    """Uk^T q . c is q . Uk c, and the values' expansion can follow the weighted sum: the form that attends over the cached
    rows themselves."""
    cfg = M.CONFIGS["lat"]
    m, eps = cfg["layers"][0]["mixer"], 1e-5
    w = {k: np.asarray(v, dtype=np.float64) for k, v in M.make_weights(cfg, 2).items()}
    x = np.random.default_rng(0).standard_normal((30, cfg["width"]))
    y = G.latent_attention(m, w, "l0.mix.", x, eps)
    H, D, R, Dv, C = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    q = (x @ w["l0.mix.q"].T).reshape(30, H, D + R)
    down = x @ w["l0.mix.dkv"].T
    c = G.rms_unit(down[:, :C], eps) * w["l0.mix.dkv.norm"]
    uk, uv = w["l0.mix.uk"].reshape(H, D, C), w["l0.mix.uv"].reshape(H, Dv, C)
    o = np.zeros((30, H, Dv))
    for i in range(30):
        js = [j for j in range(30) if G.in_window(i, j, m["mask"]["size"])]
        for a in range(H):
            qr = G.rotate_half(q[i, a, D:], i, m["rot"]["base"], R)
            s = np.array([(uk[a].T @ q[i, a, :D]) @ c[j] + qr @ G.rotate_half(down[j, C:], j, m["rot"]["base"], R) for j in js]) * m["scale"]
            o[i, a] = uv[a] @ (G.softmax(s) @ c[js])
    assert np.allclose(y, o.reshape(30, -1) @ w["l0.mix.o"].T)


def test_values_of_the_first_mixing_layer_reach_the_later_ones():
    cfg = M.CONFIGS["mix"]
    w = {k: np.asarray(v, dtype=np.float64) for k, v in M.make_weights(cfg, 4).items()}
    toks = [5, 9, 60, 3, 3, 41]
    base = G.forward(cfg, w, toks)
    full = dict(w)
    full["l3.mix.vmix"], full["l4.mix.vmix"] = np.float64(1.0), np.float64(1.0)
    changed = dict(full)
    changed["l3.mix.v"] = 5.0 * w["l3.mix.v"]                  # with lambda = 1 a later layer's own values do not matter
    assert np.allclose(G.forward(cfg, full, toks), G.forward(cfg, changed, toks)) and not np.allclose(base, G.forward(cfg, full, toks))
    none = dict(w)
    none["l3.mix.vmix"] = none["l4.mix.vmix"] = np.float64(0.0)
    off = copy.deepcopy(cfg)
    for i in (1, 3, 4):
        off["layers"][i]["mixer"]["v_mix"] = False
    assert np.allclose(G.forward(cfg, none, toks), G.forward(off, w, toks))


def test_the_mixture_is_picked_by_the_tokens_id():
    cfg = M.CONFIGS["experts"]
    w = {k: v if np.asarray(v).dtype == np.int32 else np.asarray(v, dtype=np.float64) for k, v in M.make_weights(cfg, 5).items()}
    x = np.random.default_rng(1).standard_normal((4, cfg["width"]))
    y = G.mixture(cfg["layers"][0]["mlp"], w, "l0.mlp.", x, [7, 7, 30, 8])
    for t, tok in enumerate([7, 7, 30, 8]):
        ref = G.expert(w, "l0.mlp.shared.", x[t])
        for e in w["l0.mlp.table"][tok]:
            ref = ref + G.expert(w, f"l0.mlp.e{e}.", x[t]) / 3
        assert np.allclose(y[t], ref)
    assert G.mixture(cfg["layers"][1]["mlp"], w, "l1.mlp.", x, [1, 2, 3, 4]).shape == x.shape
