"""Random Sobezen configurations — number and order of layers, head counts and sizes, ranks, which layer reads whose rows,
rotations with and without stretched frequencies, bounds, constants and weights drawn per seed — with randomly cut traces, in
both types against the plain implementation (GPU).  The second family draws sizes that the fast kernels take."""
import numpy as np
import pytest

import helpers as H
import plain_sobezen as G
import sobezen_models as M

pytestmark = pytest.mark.gpu
STORAGE = {"float32": "F32", "bfloat16": "BF16"}


def random_config(rng, fast):
    if fast:
        width, dims, inners, ranks = int(rng.choice([64, 128, 192, 256])), [16, 32, 48, 64, 96, 128], [64, 128, 192], [64, 128, 192, 256]
        rots = [16, 32, 64]
    else:
        width, dims, inners, ranks = int(rng.choice([20, 36, 48, 50, 72, 100])), [3, 4, 6, 8, 10, 16, 24, 32, 48, 80], [8, 12, 22, 40, 64], [5, 16, 24, 36, 70]
        rots = [2, 4, 6, 8, 16]
    layers, own = [], []
    for i in range(int(rng.integers(1, 6 if fast else 8))):
        kind = rng.choice(["lat", "delta", "att"], p=[0.45, 0.3, 0.25])
        if kind == "lat":
            scaling = (float(rng.uniform(1.5, 20)), float(rng.integers(20, 300)), float(rng.uniform(4, 32)), float(rng.uniform(0.5, 2))) if rng.random() < 0.6 else None
            rank, rot, base, source = int(rng.choice(ranks)), int(rng.choice(rots)), float(rng.choice([50.0, 10000.0, 1000000.0])), None
            if own and rng.random() < 0.5:
                source = int(rng.choice(own))
                m = layers[source][0][1]
                rank, rot, base = m["kv_rank"], m["rot_dim"], m["rot"]["base"]
                scaling = tuple(m["rot"]["scaling"][k] for k in ("factor", "original", "fast", "slow")) if "scaling" in m["rot"] else None
            else:
                own.append(i)
            dim = int(rng.choice(dims))
            mixer = M.lat(int(rng.integers(1, 20 if fast else 7)), dim, rot, int(rng.choice(dims)), rank, int(rng.choice(ranks)), base=base, scaling=scaling,
                          scale=float(rng.uniform(0.7, 1.5)) * (dim + rot) ** -0.5, kv_from=source)
        elif kind == "delta":
            kv = int(rng.integers(1, 4))
            mixer = M.delta(kv * int(rng.integers(1, 4)), kv, int(rng.choice(dims)), int(rng.choice(dims)), int(rng.integers(1, 6)))
        else:
            kv, dim = int(rng.integers(1, 4)), int(rng.choice([d for d in dims if d % 2 == 0]))
            mixer = M.att(kv * int(rng.integers(1, 5)), kv, dim, rot=int(rng.integers(0, dim // 2 + 1)) * 2, base=float(rng.choice([100.0, 10000.0])))
        layers.append((mixer, M.ff(int(rng.choice(inners)), rng.uniform(0.3, 6.0)) if rng.random() < 0.7 else None))
    return M.config(width, int(rng.integers(30, 400)), layers, eps=float(rng.choice([1e-6, 1e-5, 1e-3])), scale=float(rng.choice([1.0, 5.5, 0.3])),
                    logit_scale=float(rng.choice([1.0, 0.2, 3.0])))


def run(cfg, rng, seed, dtype, lengths, folder):
    import llmi_b200 as L
    w = M.write_model(folder, cfg, M.make_weights(cfg, seed, keep_state=bool(seed % 2)), STORAGE[dtype])
    model = L.load(folder, dtype)
    reqs = {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(lengths)}
    refs = {r: G.forward(cfg, w, t) for r, t in reqs.items()}
    cuts = [H.trace_whole(reqs), H.trace_portions(reqs, int(rng.integers(2, 70)), n_last=int(rng.integers(1, 20))),
            H.trace_last_decoded(reqs, n_last=int(rng.integers(20, 60))),
            H.trace_batches(reqs, int(rng.integers(2, 5)), {r: int(rng.integers(1, len(t) + 1)) for r, t in reqs.items()}),
            H.trace_mixed(reqs, {r: int(rng.integers(1, len(t) + 1)) for r, t in reqs.items()},
                          {r: int(rng.choice([1, 1, 2, 9])) for r in reqs})]
    for steps, most in cuts:
        got = H.collect(steps, H.replay(model, steps, most), cfg["vocab"])
        errs = []
        for r in refs:
            assert np.isfinite(got[r]).all(), (cfg, r)
            errs.extend((np.abs(got[r] - refs[r]).max(axis=1) / np.abs(refs[r]).max()).tolist())
        e, deep = np.asarray(errs), len(cfg["layers"]) ** 0.5
        if dtype == "float32":
            assert e.max() < 5e-5, (cfg, float(e.max()))
        else:      # bf16 rounds every layer's activations to 2^-9 of their size: bounds that grow with the root of the depth
            assert float(np.median(e)) < 1.5e-2 * deep and float(np.quantile(e, 0.9)) < 5e-2 * deep, (
                cfg, float(np.median(e)), float(np.quantile(e, 0.9)), float(e.max()))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(8))
def test_random_configuration_and_trace(seed, dtype, tmp_path):
    rng = np.random.default_rng(7100 + seed)
    cfg = random_config(rng, fast=False)
    lengths = [int(n) for n in rng.integers(1, 150, 4)] + [int(rng.choice([63, 64, 65, 128, 129]))]
    run(cfg, rng, seed, dtype, lengths, str(tmp_path / "m"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(6))
def test_random_configuration_at_the_fast_kernels_sizes(seed, dtype, tmp_path):
    rng = np.random.default_rng(7200 + seed)
    cfg = random_config(rng, fast=True)
    lengths = [int(rng.integers(130, 330)), int(rng.choice([255, 256, 257]))]
    run(cfg, rng, seed, dtype, lengths, str(tmp_path / "m"))
