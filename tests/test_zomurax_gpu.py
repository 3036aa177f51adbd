"""The Zomurax design in the library against the plain implementation of tests/plain_zomurax.py (GPU).

Every mechanism alone and together, however the work is cut: whole prompts, token by token, portions down to two
tokens, unequal batches, slots and pages that are used again (caches are poisoned with NaN before a replay), lengths at
page borders and windows' edges, the first tokens, long decoding, greedy generation through the library's own entry point.
32-bit runs must agree with the float64 oracle row by row; bf16 runs agree to bf16's precision.
"""
import math

import numpy as np
import pytest

import helpers as H
import plain_zomurax as G
import zomurax_models as M

pytestmark = pytest.mark.gpu

TOL32 = 3e-5
TOL16 = 5e-2
STORAGE = {"float32": "F32", "bfloat16": "BF16"}
LENGTHS = [1, 2, 3, 5, 31, 63, 64, 65, 100, 129, 200]


def requests_for(cfg, lengths=LENGTHS, seed=5):
    rng = np.random.default_rng(seed)
    return {f"r{i}": rng.integers(0, cfg["vocab"], n).tolist() for i, n in enumerate(lengths)}


@pytest.fixture(scope="module")
def loaded(tmp_path_factory):
    import llmi_b200 as L
    made = {}

    def get(name, dtype, lengths=LENGTHS):
        key = (name, dtype, tuple(lengths))
        if key not in made:
            cfg = M.CONFIGS[name]
            d = str(tmp_path_factory.mktemp(f"zomurax_{name}_{dtype}"))
            w = M.write_model(d, cfg, M.make_weights(cfg, 7), STORAGE[dtype])
            reqs = requests_for(cfg, lengths)
            refs = {r: G.forward(cfg, w, t) for r, t in reqs.items()}
            made[key] = (L.load(d, dtype), reqs, refs, cfg, w)
        return made[key]
    return get


def check(got, refs, dtype):
    assert set(got) == set(refs)
    errs = []
    for r in refs:
        assert got[r].shape == refs[r].shape
        assert np.isfinite(got[r]).all(), f"{r}: non-finite logits (something outside the sequence's own positions was read)"
        err = np.abs(got[r] - refs[r]).max(axis=1) / np.abs(refs[r]).max()
        if dtype == "float32":
            assert err.max() < TOL32, (r, int(err.argmax()), float(err.max()))
        errs.extend(err.tolist())
    if dtype != "float32":      # no router here whose choice could flip: every row is bounded
        e = np.asarray(errs)
        assert float(np.median(e)) < TOL16 / 2 and float(np.quantile(e, 0.98)) < TOL16 and float(e.max()) < 3 * TOL16, (
            float(np.median(e)), float(np.quantile(e, 0.98)), float(e.max()))


ALL = list(M.CONFIGS)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ALL)
def test_whole_prompts(loaded, name, dtype):
    model, reqs, refs, _, _ = loaded(name, dtype)
    steps, most = H.trace_whole(reqs)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ALL)
def test_prompt_then_token_by_token(loaded, name, dtype):
    """Most of a request in one step, its last 40 tokens one by one: windows move on under decoded tokens."""
    model, reqs, refs, _, _ = loaded(name, dtype)
    steps, most = H.trace_last_decoded(reqs, n_last=40)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


@pytest.mark.parametrize("portion", [2, 3, 7, 64, 100])
@pytest.mark.parametrize("name", ["unaligned", "att", "mix", "lat", "lat_bare", "experts", "mixed", "wide"])
def test_prompts_in_portions(loaded, name, portion):
    model, reqs, refs, _, _ = loaded(name, "float32")
    if portion < 7:
        reqs = {r: t for r, t in reqs.items() if len(t) <= 70}
    steps, most = H.trace_portions(reqs, portion, n_last=3)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), {r: refs[r] for r in reqs}, "float32")


@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_prompts_in_portions_bf16(loaded, name):
    model, reqs, refs, _, _ = loaded(name, "bfloat16")
    steps, most = H.trace_portions(reqs, 33, n_last=3)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["unaligned", "mix", "lat", "experts", "mixed", "wide", "odd"])
def test_unequal_batches_one_after_another(loaded, name, dtype):
    """Batches of four requests of unequal lengths, prompts of unequal parts of them, decoded together; the next batch
    takes the slots and pages that the one before gave back."""
    model, reqs, refs, _, _ = loaded(name, dtype)
    prompt_lens = {r: max(1, len(t) * (i % 3 + 1) // 4) for i, (r, t) in enumerate(reqs.items())}
    steps, most = H.trace_batches(reqs, 4, prompt_lens)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


@pytest.mark.parametrize("name", ["att", "lat", "experts", "mixed", "wide"])
def test_portions_beside_decoding(loaded, name):
    model, reqs, refs, _, _ = loaded(name, "float32")
    ids = list(reqs)
    first = {r: max(1, len(reqs[r]) // 3) for r in ids}
    portion = {r: (1, 5, 2, 33)[i % 4] for i, r in enumerate(ids)}
    steps, most = H.trace_mixed(reqs, first, portion)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(loaded, dtype):
    """Two tokens of prompt, then 300 steps of one token: pages are taken at 64, 128, ..., the windows' pages go back to
    the pool and are handed out again."""
    model, reqs, refs, _, _ = loaded("mixed", dtype, lengths=[302, 150])
    steps, most = H.trace_batches(reqs, 2, {r: 2 for r in reqs})
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


def test_a_windows_pages_go_back_to_the_pool(loaded):
    """A cache far smaller than the sequence in the windowed groups: decoding goes on for as long as the window's pages do."""
    model, *_ = loaded("lat", "float32")
    cache = model.new_cache(64 * 6)
    slot = cache.alloc_slot()
    import llmi_b200 as L
    for t in range(350):
        model.step(cache, [L.SequenceStep(slot, [t % 97], [])])
    windows = {g.request.window: g for g in cache.kv_groups}
    assert set(windows) == {17, 64}
    for w, g in windows.items():
        held = g.pool.n_pages - g.pool.n_free
        assert held <= (w + 63) // 64 + 1
    cache.free_slot(slot)
    cache.check()


@pytest.mark.parametrize("name", ["experts", "wide", "mixed"])
def test_greedy_generation_through_the_entry_point(loaded, name):
    """generate(): the scheduler's batches, recorded decode steps, the device's argmax — against the oracle's greedy loop."""
    import llmi_b200 as L
    model, _, _, cfg, w = loaded(name, "float32")
    rng = np.random.default_rng(3)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (1, 9, 70, 4, 33)]
    new = [12, 5, 12, 1, 9]
    out = L.generate(model, prompts, max_new=new, max_batch=3)
    ref = [G.greedy(cfg, w, p, n) for p, n in zip(prompts, new)]
    assert out == ref
    assert L.generate(model, prompts, max_new=new, max_batch=3, use_graphs=False) == ref


def test_recorded_steps_in_bf16_follow_the_plain_steps(loaded):
    """bf16 serving pads and records its steps (decode graphs, padded prompt steps): generation with and without them
    gives the same tokens, three times over (from the second time on everything is replayed)."""
    import llmi_b200 as L
    model, _, _, cfg, _ = loaded("wide", "bfloat16")
    assert model.pads_prompts
    rng = np.random.default_rng(9)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (3, 40, 130, 17)]
    plain = L.generate(model, prompts, max_new=20, max_batch=4, use_graphs=False)
    for _ in range(3):
        assert L.generate(model, prompts, max_new=20, max_batch=4) == plain


def test_sampling_takes_the_capped_logits(loaded):
    """The cap changes no order but every probability: with a temperature the tokens follow the capped logits."""
    model, reqs, refs, cfg, _ = loaded("wide", "float32")
    import llmi_b200 as L
    cache = model.new_cache(256)
    slot = cache.alloc_slot()
    out = model.step(cache, [L.SequenceStep(slot, reqs["r8"], [99])]).cpu().numpy()[0]
    assert np.abs(out).max() < cfg["logit_softcap"] and np.abs(out - refs["r8"][99]).max() < 1e-3
    cache.free_slot(slot)


def test_programs_as_a_user_calls_them(tmp_path):
    """bin/llmi-generate and bin/trace_run on a Zomurax folder, as subprocesses: the design is chosen by config.json."""
    import json
    import os
    import subprocess
    import sys
    from conftest import ROOT
    cfg = M.CONFIGS["experts"]
    d = str(tmp_path / "model")
    w = M.write_model(d, cfg, M.make_weights(cfg, 7), "F32")
    prompt = [3, 17, 80, 4, 4, 56]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "llmi-generate"), d, "--ids", ",".join(map(str, prompt)),
                        "--max-new", "6", "--json", "--dtype", "fp32"], capture_output=True, text=True, timeout=200)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[-1])["generated_ids"] == G.greedy(cfg, w, prompt, 6)
    reqs = requests_for(cfg, [5, 70, 33])
    steps, _ = H.trace_batches(reqs, 3, {"r0": 2, "r1": 40, "r2": 33})
    out = tmp_path / "out"
    most = sum(len(t) for t in reqs.values())
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", d, "--dtype", "float32",
                        "--out", str(out), "--max-tokens", str(most)],
                       input="".join(json.dumps(s_) + "\n" for s_ in steps), capture_output=True, text=True, timeout=200)
    assert p.returncode == 0, p.stderr[-2000:]
    outs = []
    for s_ in steps:
        n = sum(len(e["want"]) for e in s_["entries"])
        outs.append(np.fromfile(out / f"{s_['step']}.f32", dtype="<f4").reshape(n, -1) if n else None)
    check(H.collect(steps, outs, cfg["vocab"]), {r: G.forward(cfg, w, t) for r, t in reqs.items()}, "float32")


def test_a_table_that_names_no_expert_is_refused(tmp_path):
    import llmi_b200 as L
    cfg = M.CONFIGS["experts"]
    w = M.make_weights(cfg, 1)
    w["l0.mlp.table"][5, 1] = 5
    M.write_model(str(tmp_path / "m"), cfg, w, "F32")
    with pytest.raises(ValueError, match="table"):
        L.load(str(tmp_path / "m"), "float32")


# ----------------------------------------------------------------------------- kernels alone

class _Ctx:
    pass


def _ctx(q_lens, first_pos):
    """The index arrays of a step in which sequence s brings ``q_lens[s]`` tokens from position ``first_pos[s]`` on."""
    import torch
    ctx = _Ctx()
    ctx.decode = all(n == 1 for n in q_lens)
    ctx.n_seqs = ctx.n_real_seqs = len(q_lens)
    dev = "cuda:0"
    ctx.tok_seq = torch.tensor(np.repeat(np.arange(len(q_lens)), q_lens).astype(np.int32), device=dev)
    ctx.tok_pos = torch.tensor(np.concatenate([np.arange(p, p + n) for p, n in zip(first_pos, q_lens)]).astype(np.int32), device=dev)
    ctx.seq_q_start = torch.tensor(np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int32), device=dev)
    ctx.seq_kv_len = torch.tensor([p + n for p, n in zip(first_pos, q_lens)], dtype=torch.int32, device=dev)
    ctx.host_q_lens, ctx.host_kv_lens = list(q_lens), [p + n for p, n in zip(first_pos, q_lens)]
    return ctx


def _paged(rows, order, page, dt, dead=()):
    """rows [N, heads, d] -> a cache tensor [pages, heads, page, d] with the sequence's pages at ``order``; everything
    else, and the pages numbered in ``dead``, NaN."""
    import torch
    N, heads, d = rows.shape
    cache = torch.full((int(max(order)) + 2, heads, page, d), float("nan"), dtype=dt, device="cuda:0")
    for i, pg in enumerate(order):
        lo, hi = i * page, min((i + 1) * page, N)
        if hi > lo and i not in dead:
            cache[pg, :, :hi - lo] = rows[lo:hi].permute(1, 0, 2).to("cuda:0")
    return cache


def _attention_reference(q, k, v, scale, window, r1, r2, sink, rows):
    """q [N, H, dk], k [N, G, dk], v [N, G, dv] float64 -> [len(rows), H, dv] for the queries at ``rows``."""
    Hq, Gk = q.shape[1], k.shape[1]
    out = np.zeros((len(rows), Hq, v.shape[2]))
    for n, t in enumerate(rows):
        js = np.array([j for j in range(t + 1) if G.in_window(t, j, window)])
        for h in range(Hq):
            g = h // (Hq // Gk)
            s = k[js, g] @ q[t, h] * scale - (G.distance_bias((t - js).astype(float), r1[h], r2[h]) if r1 is not None else 0.0)
            out[n, h] = G.softmax(s, None if sink is None else sink[h]) @ v[js, g]
    return out


SIZES = [(2, 1, 16, 16), (4, 2, 96, 48), (4, 1, 64, 64), (2, 2, 128, 128), (8, 2, 128, 32), (6, 2, 24, 40), (3, 3, 10, 7), (4, 2, 48, 128)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", SIZES)
@pytest.mark.parametrize("window,key", [(0, 0), (0, 63), (0, 64), (0, 191), (0, 255), (0, 256), (0, 298), (0, 299),
                                        (100, 199), (100, 200), (64, 235), (64, 236), (1, 298), (1, 299), (300, 0), (299, 0), (299, 1)])
def test_attention_with_a_bias_by_distance_and_a_sink(window, key, sizes, dtype):
    """300 cached positions on pages that are not in order, one position (``key``) made to stand out for the last head by
    scaling it and the query, by far more than its distance costs and the sink takes.  The query at 299 — a single token,
    and the last of portions of 70 and 200 tokens — must return that position's own value row when it sees it, and must
    not see it otherwise; every row is compared with the plain sums, where the other heads' biases (from nearly none to
    steep) and sinks decide."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.ops import kernels
    Hq, Gk, dk, dv = sizes
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(key + 7 * window)
    N, page, scale = 300, 64, 0.5
    k = torch.tensor(rng.standard_normal((N, Gk, dk)).astype(np.float32)).to(dt)
    v = torch.tensor(rng.standard_normal((N, Gk, dv)).astype(np.float32)).to(dt)
    q = torch.tensor((rng.standard_normal((N, Hq, dk)) * 4 / math.sqrt(dk)).astype(np.float32))
    others = np.arange(N) != key
    k[others, Gk - 1] *= 0.1
    q[:, -1] = k[key, Gk - 1].float() * (80.0 / dk)      # the score of `key` for the last head: about 40
    q = q.to(dt)
    r1 = rng.uniform(0.02, 2.5, Hq).astype(np.float32)
    r2 = rng.uniform(0.05, 0.6, Hq).astype(np.float32)
    sink = rng.uniform(-1.0, 5.0, Hq).astype(np.float32)
    order = rng.permutation(9)[:5]
    rt = Runtime(dt, "cuda:0")
    pages = torch.tensor(order[None, :].astype(np.int32), device="cuda:0")
    dead = [i for i in range(5) if window and (i + 1) * page <= N - 200 - window + 1]       # pages that no query here sees
    kc, vc = _paged(k, order, page, dt, dead), _paged(v, order, page, dt, dead)
    kk, vv, qq = (x.float().numpy().astype(np.float64) for x in (k, v, q))
    ref = _attention_reference(qq, kk, vv, scale, window, r1.astype(float), r2.astype(float), sink.astype(float), list(range(N - 200, N)))
    plain = _attention_reference(qq, kk, vv, scale, window, None, None, sink.astype(float), [N - 1])
    dev = {n: torch.tensor(a, device="cuda:0") for n, a in (("r1", r1), ("r2", r2), ("sink", sink))}
    tol = 2e-5 if dtype == "float32" else 3e-2
    for n_rows in (1, 70, 200):
        ctx = _ctx([n_rows], [N - n_rows])
        out = torch.full((n_rows, Hq * dv), float("nan"), dtype=dt, device="cuda:0")
        qd = q[N - n_rows:].reshape(n_rows, -1).to("cuda:0").contiguous()
        kernels.attention_maps(qd, out, kc, vc, ctx, pages, page, Hq, Gk, 1, dk, dv, scale, None, window, 0, rt=rt,
                               bias=(dev["r1"], dev["r2"]), sink=dev["sink"])
        kernels.check_device_errors(torch.device("cuda:0"))
        got = out.float().cpu().numpy().reshape(n_rows, Hq, dv)
        assert np.isfinite(got).all() and np.abs(got - ref[200 - n_rows:]).max() < tol, (n_rows, float(np.abs(got - ref[200 - n_rows:]).max()))
        alone = np.abs(got[-1, -1] - vv[key, Gk - 1]).max() < 0.05
        assert alone == G.in_window(299, key, window), (key, window)
        if n_rows == 1:      # a sink without a bias
            kernels.attention_maps(qd, out, kc, vc, ctx, pages, page, Hq, Gk, 1, dk, dv, scale, None, window, 0, rt=rt, sink=dev["sink"])
            assert np.abs(out.float().cpu().numpy().reshape(1, Hq, dv) - plain).max() < tol


@pytest.mark.parametrize("sizes", [(2, 1, 64, 64), (2, 2, 128, 128), (4, 2, 96, 48)])
def test_attention_over_a_long_context_that_is_cut_over_positions(sizes):
    """2,500 positions: a prompt block's key range is cut into jobs and single tokens' positions into parts; the sink
    counts once however many parts there are, and a far key at a distance of more than two thousand stands out."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.ops import kernels
    Hq, Gk, dk, dv = sizes
    rng = np.random.default_rng(dk)
    N, page, scale, dt, key = 2500, 64, 0.5, torch.bfloat16, 130
    k = torch.tensor(rng.standard_normal((N, Gk, dk)).astype(np.float32)).to(dt)
    v = torch.tensor(rng.standard_normal((N, Gk, dv)).astype(np.float32)).to(dt)
    q = torch.tensor((rng.standard_normal((N, Hq, dk)) * 2 / math.sqrt(dk)).astype(np.float32))
    k[np.arange(N) != key, Gk - 1] *= 0.1
    q[-40:, -1] = k[key, Gk - 1].float() * (80.0 / dk)
    q = q.to(dt)
    r1, r2, sink = np.array([0.3] * (Hq - 1) + [1.0], np.float32), np.array([0.01] * Hq, np.float32), np.array([6.0] * Hq, np.float32)
    order = rng.permutation(50)[:40]
    rt = Runtime(dt, "cuda:0")
    pages = torch.tensor(order[None, :].astype(np.int32), device="cuda:0")
    kc, vc = _paged(k, order, page, dt), _paged(v, order, page, dt)
    kk, vv, qq = (x.float().numpy().astype(np.float64) for x in (k, v, q))
    rows = [1500, 1627, 1628, 2000, 2460, 2498, 2499]
    ref = _attention_reference(qq, kk, vv, scale, 0, r1.astype(float), r2.astype(float), sink.astype(float), rows)
    dev = [torch.tensor(a, device="cuda:0") for a in (r1, r2, sink)]
    for n_rows in (1, 1000):
        ctx = _ctx([n_rows], [N - n_rows])
        out = torch.full((n_rows, Hq * dv), float("nan"), dtype=dt, device="cuda:0")
        kernels.attention_maps(q[N - n_rows:].reshape(n_rows, -1).to("cuda:0").contiguous(), out, kc, vc, ctx, pages, page, Hq, Gk, 1, dk, dv,
                               scale, None, 0, 0, rt=rt, bias=(dev[0], dev[1]), sink=dev[2])
        kernels.check_device_errors(torch.device("cuda:0"))
        got = out.float().cpu().numpy().reshape(n_rows, Hq, dv)
        for n, t in enumerate(rows):
            if t >= N - n_rows:
                assert np.abs(got[t - (N - n_rows)] - ref[n]).max() < 2e-2, (n_rows, t)
        assert np.abs(got[-1, -1] - vv[key, Gk - 1]).max() < 0.05


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("Hq,C,R", [(5, 28, 8), (3, 64, 16), (16, 128, 64), (20, 512, 64), (2, 96, 0), (6, 192, 32)])
@pytest.mark.parametrize("window,key", [(0, 0), (0, 299), (100, 199), (100, 200), (64, 235), (64, 236), (65, 234), (65, 235), (1, 298), (1, 299), (300, 0), (299, 0), (150, 150), (150, 149)])
def test_latent_attention_over_a_window(window, key, Hq, C, R, dtype):
    """The same with one cached row for all heads: pages before every window are NaN, the key's row stands out for the last
    head only."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.ops import kernels
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(key + window + C)
    N, page, scale, D = 300, 64, 0.5, C + R
    rows = torch.tensor((rng.standard_normal((N, 1, D)) * 0.5).astype(np.float32))
    rows[np.arange(N) != key] *= 0.1
    rows = rows.to(dt)
    q = torch.tensor((rng.standard_normal((N, Hq, D)) * 8 / math.sqrt(D)).astype(np.float32))
    q[:, -1] = rows[key, 0].float() * (320.0 / D)
    q = q.to(dt)
    order = rng.permutation(9)[:5]
    rt = Runtime(dt, "cuda:0")
    pages = torch.tensor(order[None, :].astype(np.int32), device="cuda:0")
    kk, qq = rows.float().numpy().astype(np.float64), q.float().numpy().astype(np.float64)
    ref = _attention_reference(qq, kk, kk[..., :C], scale, window, None, None, None, list(range(N - 200, N)))
    tol = 2e-5 if dtype == "float32" else 2e-2
    for n_rows in (1, 70, 200):
        dead = [i for i in range(5) if window and (i + 1) * page <= N - n_rows - window + 1]
        table = pages.clone()
        table[0, dead] = -1                                            # (given back)
        cache = _paged(rows, order, page, dt, dead)
        ctx = _ctx([n_rows], [N - n_rows])
        out = torch.full((n_rows, Hq * C), float("nan"), dtype=dt, device="cuda:0")
        kernels.attention_latent(q[N - n_rows:].reshape(n_rows, -1).to("cuda:0").contiguous(), out, cache, ctx, table, page, Hq, C, R, scale,
                                 rt=rt, window=window)
        got = out.float().cpu().numpy().reshape(n_rows, Hq, C)
        assert np.isfinite(got).all() and np.abs(got - ref[200 - n_rows:]).max() < tol, (n_rows, float(np.abs(got - ref[200 - n_rows:]).max()))
        alone = np.abs(got[-1, -1] - kk[key, 0, :C]).max() < 0.05
        assert alone == G.in_window(299, key, window), (key, window)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("Hq,Gk,dk,dv", [(4, 2, 64, 32), (5, 1, 6, 7), (2, 2, 132, 256), (3, 3, 20, 12)])
@pytest.mark.parametrize("temp", [None, (0.7, 5), (0.3, 1)])
def test_unit_heads_temperature_and_mixed_values(Hq, Gk, dk, dv, temp, dtype):
    """Two sequences, one of them going on from position 61 across a page's border: q into its buffer, k and v into their
    cache rows; values plain, kept for later layers, and mixed with what was kept."""
    import torch
    from llmi_b200.ops import kernels
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(Hq + dk)
    lens, starts, eps, lam, page = [9, 7], [61, 0], 1e-3, 0.3, 64
    T, n_in = sum(lens), Hq * dk + Gk * (dk + dv)
    proj = (rng.standard_normal((T, n_in + 4)) * 0.2).astype(np.float32)
    ctx = _ctx(lens, starts)
    pos = ctx.tok_pos.cpu().numpy()
    pages = torch.tensor([[3, 1], [0, -1]], dtype=torch.int32, device="cuda:0")
    first = torch.full((T, Gk * dv), float("nan"), device="cuda:0")
    q_ref = G.rms_unit(proj[:, :Hq * dk].reshape(T, Hq, dk).astype(np.float64), eps)
    if temp:
        q_ref = q_ref * np.array([G.temperature(p, *temp) for p in pos])[:, None, None]
    k_ref = G.rms_unit(proj[:, Hq * dk:(Hq + Gk) * dk].reshape(T, Gk, dk).astype(np.float64), eps)
    v_own = proj[:, (Hq + Gk) * dk:n_in].astype(np.float64)
    kept = rng.standard_normal((T, Gk * dv)).astype(np.float32)
    tol = 1e-5 if dtype == "float32" else 1.5e-2
    for mode in (kernels.VALUES_PLAIN, kernels.VALUES_KEEP, kernels.VALUES_MIX):
        kc = torch.full((5, Gk, page, dk), float("nan"), dtype=dt, device="cuda:0")
        vc = torch.full((5, Gk, page, dv), float("nan"), dtype=dt, device="cuda:0")
        q = torch.full((T, Hq * dk), float("nan"), dtype=dt, device="cuda:0")
        if mode == kernels.VALUES_MIX:
            first.copy_(torch.tensor(kept))
        kernels.qkv_unit_prepare(torch.tensor(proj, device="cuda:0")[:, :n_in], Hq, Gk, dk, Gk, dv, ctx, pages, page, kc, vc, q, eps, temp, mode,
                                 lam, first if mode else None)
        assert np.abs(q.float().cpu().numpy().reshape(T, Hq, dk) - q_ref).max() < tol * max(1.0, np.abs(q_ref).max())
        v_ref = G.mix_values(v_own, kept.astype(np.float64), lam) if mode == kernels.VALUES_MIX else v_own
        if mode == kernels.VALUES_KEEP:
            assert np.abs(first.cpu().numpy() - v_own).max() < 1e-6
        written = 0
        for t in range(T):
            s = 0 if t < lens[0] else 1
            pg = int(pages[s, pos[t] // page])
            assert np.abs(kc[pg, :, pos[t] % page].float().cpu().numpy() - k_ref[t]).max() < tol * 4
            assert np.abs(vc[pg, :, pos[t] % page].float().cpu().numpy() - v_ref[t].reshape(Gk, dv)).max() < tol * 4
            written += Gk * dk
        assert int((~torch.isnan(kc)).sum()) == written                  # and nothing else


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("Hq,D,C,R,dims", [(4, 16, 32, 8, 8), (3, 7, 13, 6, 4), (2, 64, 128, 64, 64), (5, 6, 9, 3, 2), (2, 8, 16, 0, 0)])
@pytest.mark.parametrize("pairing", [0, 1])
def test_queries_and_latent_straight_from_the_projected_row(Hq, D, C, R, dims, pairing, dtype):
    import torch
    from llmi_b200.ops import kernels
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(Hq + D)
    lens, starts, page, eps, base = [5, 8], [60, 0], 64, 1e-4, 300.0
    T = sum(lens)
    proj = rng.standard_normal((T, Hq * (D + R) + C + R)).astype(np.float32)
    wc = (1.0 + 0.3 * rng.standard_normal(C)).astype(np.float32)
    ctx = _ctx(lens, starts)
    pos = ctx.tok_pos.cpu().numpy()
    pages = torch.tensor([[2, 4], [1, -1]], dtype=torch.int32, device="cuda:0")
    inv = np.array([base ** (-2.0 * i / max(dims, 1)) for i in range(dims // 2)] or [0.0], np.float32)
    cache = torch.full((5, 1, page, C + R), float("nan"), dtype=dt, device="cuda:0")
    qn = torch.full((T, Hq * D), float("nan"), dtype=dt, device="cuda:0")
    qa = torch.full((T, Hq * (C + R)), float("nan"), dtype=dt, device="cuda:0")
    kernels.latent_prepare_direct(torch.tensor(proj, device="cuda:0"), Hq, D, C, R, torch.tensor(wc, device="cuda:0"), eps,
                                  torch.tensor(inv, device="cuda:0"), dims, pairing, ctx, pages, page, cache, qn, qa)
    x = proj.astype(np.float64)
    q = x[:, :Hq * (D + R)].reshape(T, Hq, D + R)

    def turn(v, p):
        if not dims:
            return v
        order = np.concatenate([np.arange(0, dims, 2), np.arange(1, dims, 2), np.arange(dims, v.shape[-1])]) if pairing else np.arange(v.shape[-1])
        y = np.empty_like(v)
        y[..., order] = G.rotate_half(v[..., order], p, base, dims)      # neighbours turn as halves of the reordered entries do
        return y
    tol = 2e-5 if dtype == "float32" else 2e-2
    assert np.abs(qn.float().cpu().numpy().reshape(T, Hq, D) - q[..., :D]).max() < tol
    got = qa.float().cpu().numpy().reshape(T, Hq, C + R)
    assert np.isnan(got[..., :C]).all()
    c = G.rms_unit(x[:, Hq * (D + R):Hq * (D + R) + C], eps) * wc
    for t in range(T):
        if R:
            assert np.abs(got[t, :, C:] - turn(q[t, :, D:], pos[t])).max() < tol
        row = cache[int(pages[0 if t < lens[0] else 1, pos[t] // page]), 0, pos[t] % page].float().cpu().numpy()
        assert np.abs(row[:C] - c[t]).max() < 2 * tol
        if R:
            assert np.abs(row[C:] - turn(x[t, -R:], pos[t])).max() < tol
    assert int((~torch.isnan(cache)).sum()) == T * (C + R)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,W", [(5, 36), (70, 256), (3, 2048), (600, 1000), (2, 50), (1, 9000)])
def test_a_norm_that_replaces_the_sum(T, W, dtype):
    import torch
    from llmi_b200.ops import kernels
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(T + W)
    x, y = (rng.standard_normal((T, W)).astype(np.float32) * s for s in (1.0, 2.0))
    g = (1.0 + 0.3 * rng.standard_normal(W)).astype(np.float32)
    tx, ty, tg = (torch.tensor(v, device="cuda:0") for v in (x, y, g))
    ref = G.rms_unit(2.5 * x.astype(np.float64) + y, 1e-3) * g
    x1, h = tx.clone(), torch.full((T, W), float("nan"), dtype=dt, device="cuda:0")
    kernels.stream_postnorm(x1, ty, 2.5, tg, 1e-3, h)
    assert np.abs(x1.cpu().numpy() - ref).max() < 1e-5
    assert torch.equal(h, x1.to(dt))
    x2 = tx.clone()
    kernels.stream_postnorm(x2, ty, 2.5, tg, 1e-3)
    assert torch.equal(x1, x2)
    kernels.stream_postnorm(tx, None, 1.0, None, 0.0, h)
    assert torch.equal(h, tx.to(dt)) and np.array_equal(tx.cpu().numpy(), x)


def test_capped_rows_and_experts_by_the_tokens_id():
    import torch
    from llmi_b200.ops import kernels
    rng = np.random.default_rng(0)
    z = (rng.standard_normal((7, 333)) * 40).astype(np.float32)
    t = torch.tensor(z, device="cuda:0")
    kernels.softcap_rows(t, 9.0)
    assert np.abs(t.cpu().numpy() - 9.0 * np.tanh(z.astype(np.float64) / 9.0)).max() < 1e-5
    table = torch.tensor(rng.integers(0, 20, (50, 3)).astype(np.int32), device="cuda:0")
    ctx = _ctx([30, 5], [0, 9])
    ctx.tok_seq[4] = -1
    ids = torch.tensor(rng.integers(0, 50, 35).astype(np.int32), device="cuda:0")
    ids[4] = -1
    idx = torch.zeros((35, 3), dtype=torch.int32, device="cuda:0")
    wt = torch.zeros((35, 3), device="cuda:0")
    kernels.moe_table(table, ids, ctx, idx, wt)
    live = torch.arange(35, device="cuda:0") != 4
    assert torch.equal(idx[live], table[ids[live].long()]) and (idx[4] == -1).all() and (wt[4] == 0).all()
    assert torch.allclose(wt[live], torch.full((34, 3), 1 / 3, device="cuda:0"))


@pytest.mark.parametrize("act", ["silu", "gelu_tanh"])
@pytest.mark.parametrize("T,E,top,W,F", [(3, 4, 2, 64, 48), (300, 5, 3, 136, 72), (600, 4, 2, 128, 128), (1500, 8, 2, 256, 200), (1024, 3, 1, 192, 136), (700, 12, 3, 512, 64)])
def test_gated_experts_on_every_kind_of_tile(T, E, top, W, F, act):
    """Streamed weights (a few tokens), mma.sync tiles, tcgen05 tiles (from 1,024 items and 128 rows on, gate and up rows in
    turn): the same sum, with token rows of no sequence and one expert that nobody picks; rows of the up matrices that lie
    ahead of the gate matrices in memory take the other tiles."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.ops import kernels
    rt = Runtime(torch.bfloat16, "cuda:0")
    gen = torch.Generator(device="cuda:0").manual_seed(T + E)

    def rnd(*shape, gain=1.0):
        return (torch.randn(*shape, generator=gen, device="cuda:0") * gain).to(torch.bfloat16)
    h, both, wd = rnd(T, W), rnd(2, E, F, W, gain=2 * W ** -0.5), rnd(E, W, F, gain=F ** -0.5)
    score = torch.rand(T, E, generator=gen, device="cuda:0")
    if E > top:
        score[:, E - 2] = -1.0                                            # nobody picks it
    idx = score.topk(top, dim=1).indices.to(torch.int32).contiguous()
    idx[T // 2] = -1
    wt = torch.full((T, top), 1.0 / top, device="cuda:0")
    code = kernels.EXPERT_ACTIVATIONS[act]
    fn = torch.nn.functional.silu if act == "silu" else lambda z: torch.nn.functional.gelu(z, approximate="tanh")
    for wg, wu in ((both[0], both[1]), (both[1], both[0])):
        y = torch.full((T, W), float("nan"), device="cuda:0")
        if kernels.moe_grouped_applies(h, W, F, E):
            kernels.moe_experts_grouped(h, wg, wu, wd, idx, wt, code, rt, y)
            again = torch.ones((T, W), device="cuda:0")
            kernels.moe_experts_grouped(h, wg, wu, wd, idx, wt, code, rt, again, add=True)
            assert torch.equal(again, 1.0 + y)
        else:
            kernels.moe_experts_streamed(h, wg, wu, wd, idx, wt, code, torch.empty((T, top, F), device="cuda:0"), y)
        kernels.check_device_errors(torch.device("cuda:0"))
        hd, ref = h.double(), torch.zeros((T, W), dtype=torch.float64, device="cuda:0")
        for e in range(E):
            for j in range(top):
                rows = (idx[:, j] == e).nonzero().flatten()
                if rows.numel():
                    a = fn(hd[rows] @ wg[e].double().T) * (hd[rows] @ wu[e].double().T)
                    ref[rows] += wt[rows, j].double()[:, None] * (a @ wd[e].double().T)
        err = (y.double() - ref).abs().max(dim=1).values / ref.abs().max()
        assert torch.isfinite(y).all() and float(err.max()) < 1.5e-2 and float(y[T // 2].abs().max()) == 0.0, (int(err.argmax()), float(err.max()))
