"""Random Zomurax configurations — number and order of layers, head counts and sizes, windows, temperatures, which layers
mix values, experts with and without one beside them, constants and weights drawn per seed — with randomly cut traces, in
both types against the plain implementation (GPU).  The second family draws sizes that the fast kernels take (head sizes
that are multiples of 16, latents that are multiples of 64) with requests of a few hundred tokens, so that windows pass
over page borders in the fast kernels too."""
import numpy as np
import pytest

import helpers as H
import plain_zomurax as G
import zomurax_models as M

pytestmark = pytest.mark.gpu
STORAGE = {"float32": "F32", "bfloat16": "BF16"}


def random_config(rng, fast):
    if fast:
        width, dims, inners, ranks, longest = int(rng.choice([64, 128, 192, 256])), [16, 32, 48, 64, 96, 128], [64, 128, 192], [64, 128, 192, 256], 250
    else:
        width, dims, inners, ranks, longest = int(rng.choice([20, 36, 48, 50, 72, 100])), [3, 4, 6, 8, 10, 16, 24, 32, 48, 80], [8, 12, 22, 40, 64], [5, 16, 24, 36, 70], 120
    mix_heads = int(rng.integers(1, 4))                  # layers that mix have this many key/value heads of this size
    mix_dim = int(rng.choice(dims))
    layers = []
    for _ in range(int(rng.integers(1, 5 if fast else 8))):
        if rng.random() < 0.55:
            mix = bool(rng.random() < 0.7)
            kv = mix_heads if mix else int(rng.integers(1, 4))
            temp = (float(rng.uniform(-0.1, 0.8)), int(rng.integers(1, longest))) if rng.random() < 0.8 else None
            dim = int(rng.choice([64, 128] if fast and rng.random() < 0.4 else dims))
            mixer = M.att(kv * int(rng.integers(1, 5)), kv, dim, mix_dim if mix else int(rng.choice([dim] + dims)),
                          scale=float(rng.uniform(1.0, 3.0)) * dim ** -0.5, mix=mix, temp=temp)
        else:
            dim, rot = int(rng.choice(dims)), int(rng.choice([r for r in (0, 2, 4, 8, 16, 32, 64) if not fast or r % 16 == 0]))
            mixer = M.lat(int(rng.integers(1, 20 if fast else 7)), dim, rot, int(rng.choice(dims)), int(rng.choice(ranks)),
                          int(rng.integers(1, longest)) if rng.random() < 0.85 else None, base=float(rng.choice([50.0, 10000.0, 1000000.0])),
                          scale=float(rng.uniform(0.7, 1.5)) * (dim + rot) ** -0.5)
        mlp = None
        if rng.random() < 0.8:
            experts = int(rng.integers(1, 13))
            mlp = M.moe(int(rng.choice(inners)), experts, int(rng.integers(1, min(experts, 5) + 1)),
                        shared=int(rng.choice(inners)) if rng.random() < 0.7 else None)
        layers.append((mixer, mlp))
    return M.config(width, int(rng.integers(30, 400)), layers, eps=float(rng.choice([1e-6, 1e-5, 1e-3])),
                    alpha=float(rng.choice([0.5, 1.0, 2.0, 3.0])), cap=float(rng.choice([4.0, 15.0, 50.0])))


def run(cfg, rng, seed, dtype, lengths, folder):
    import llmi_b200 as L
    w = M.write_model(folder, cfg, M.make_weights(cfg, seed), STORAGE[dtype])
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
    rng = np.random.default_rng(9100 + seed)
    cfg = random_config(rng, fast=False)
    lengths = [int(n) for n in rng.integers(1, 150, 4)] + [int(rng.choice([63, 64, 65, 128, 129]))]
    run(cfg, rng, seed, dtype, lengths, str(tmp_path / "m"))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("seed", range(5))
def test_random_configuration_at_the_fast_kernels_sizes(seed, dtype, tmp_path):
    rng = np.random.default_rng(9200 + seed)
    cfg = random_config(rng, fast=True)
    lengths = [int(rng.integers(130, 330)), int(rng.choice([255, 256, 257]))]
    run(cfg, rng, seed, dtype, lengths, str(tmp_path / "m"))
