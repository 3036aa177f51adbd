"""The Sobezen design in the library against the plain implementation of tests/plain_sobezen.py (GPU).

Every mechanism alone and together, however the work is cut: whole prompts, token by token, portions down to two tokens,
unequal batches, slots, pages and states that are used again (caches are poisoned with NaN before a replay), lengths at page
borders, the first tokens, long decoding, greedy generation through the library's own entry point.  32-bit runs must agree
with the float64 oracle row by row; bf16 runs agree to bf16's precision.
"""
import math

import numpy as np
import pytest

import helpers as H
import plain_sobezen as G
import sobezen_models as M

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

    def get(name, dtype, lengths=LENGTHS, keep_state=False):
        key = (name, dtype, tuple(lengths), keep_state)
        if key not in made:
            cfg = M.CONFIGS[name]
            d = str(tmp_path_factory.mktemp(f"sobezen_{name}_{dtype}"))
            w = M.write_model(d, cfg, M.make_weights(cfg, 7, keep_state), STORAGE[dtype])
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
    if dtype != "float32":
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
    model, reqs, refs, _, _ = loaded(name, dtype)
    steps, most = H.trace_last_decoded(reqs, n_last=40)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


def test_the_stream_after_every_layer(loaded):
    """The residual stream behind the embedding and behind every layer, not only the logits."""
    import llmi_b200 as L
    model, reqs, _, cfg, w = loaded("mixed", "float32")
    toks = reqs["r8"]
    states = G.forward(cfg, w, toks, return_states=True)[1]
    cache = model.new_cache(256)
    trace = []
    model.step(cache, [L.SequenceStep(cache.alloc_slot(), toks, [len(toks) - 1])], trace=trace)
    for got, ref in zip(trace[1:], states):
        assert np.abs(got.cpu().numpy() - ref).max() < 3e-5 * np.abs(ref).max()


@pytest.mark.parametrize("portion", [2, 3, 7, 64, 100])
@pytest.mark.parametrize("name", ["lat", "shared", "delta", "delta_one_tap", "att", "mixed", "wide", "odd"])
def test_prompts_in_portions(loaded, name, portion):
    model, reqs, refs, _, _ = loaded(name, "float32")
    if portion < 7:
        reqs = {r: t for r, t in reqs.items() if len(t) <= 70}
    steps, most = H.trace_portions(reqs, portion, n_last=3)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), {r: refs[r] for r in reqs}, "float32")


@pytest.mark.parametrize("name", ["shared", "mixed", "wide"])
def test_prompts_in_portions_bf16(loaded, name):
    model, reqs, refs, _, _ = loaded(name, "bfloat16")
    steps, most = H.trace_portions(reqs, 33, n_last=3)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, "bfloat16")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["shared", "delta", "delta_one_tap", "gate", "mixed", "wide", "odd"])
def test_unequal_batches_one_after_another(loaded, name, dtype):
    """Batches of four requests of unequal lengths, prompts of unequal parts of them, decoded together; the next batch
    takes the slots, pages and states that the one before gave back."""
    model, reqs, refs, _, _ = loaded(name, dtype)
    prompt_lens = {r: max(1, len(t) * (i % 3 + 1) // 4) for i, (r, t) in enumerate(reqs.items())}
    steps, most = H.trace_batches(reqs, 4, prompt_lens)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


@pytest.mark.parametrize("name", ["lat", "shared", "delta", "mixed", "wide"])
def test_portions_beside_decoding(loaded, name):
    model, reqs, refs, _, _ = loaded(name, "float32")
    ids = list(reqs)
    first = {r: max(1, len(reqs[r]) // 3) for r in ids}
    portion = {r: (1, 5, 2, 33)[i % 4] for i, r in enumerate(ids)}
    steps, most = H.trace_mixed(reqs, first, portion)
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, "float32")


@pytest.mark.parametrize("cut", ["decoded", "portions", "mixed"])
@pytest.mark.parametrize("name", ["delta", "wide", "odd"])
def test_a_state_that_never_fades_through_every_cut(loaded, name, cut):
    """Decays next to one: a state or a carried convolution input that is lost, zeroed or cut anywhere changes everything
    after it."""
    model, reqs, refs, _, _ = loaded(name, "float32", keep_state=True)
    steps, most = {"decoded": lambda: H.trace_last_decoded(reqs, n_last=60), "portions": lambda: H.trace_portions(reqs, 21, n_last=5),
                   "mixed": lambda: H.trace_mixed(reqs, {r: max(1, len(t) // 2) for r, t in reqs.items()},
                                                  {r: (1, 2, 17)[i % 3] for i, r in enumerate(reqs)})}[cut]()
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, "float32")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "wide"])
def test_long_decoding(loaded, name, dtype):
    """Two tokens of prompt, then 300 steps of one token: pages are taken at 64, 128, ..., the state is carried on."""
    model, reqs, refs, _, _ = loaded(name, dtype, lengths=[302, 150])
    steps, most = H.trace_batches(reqs, 2, {r: 2 for r in reqs})
    check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


@pytest.mark.parametrize("n_seqs", [5, 17, 40])
def test_many_sequences_decode_together(loaded, n_seqs):
    """More sequences in a step of single tokens than the low-rank products take at a time (4, 8, 16), each as if alone."""
    for dtype in ("float32", "bfloat16"):
        model, _, _, cfg, w = loaded("wide", dtype)
        rng = np.random.default_rng(n_seqs)
        reqs = {f"r{i}": rng.integers(0, cfg["vocab"], 9 + i % 7).tolist() for i in range(n_seqs)}
        refs = {r: G.forward(cfg, w, t) for r, t in reqs.items()}
        steps, most = H.trace_batches(reqs, n_seqs, {r: 1 + i % 4 for i, r in enumerate(reqs)})
        check(H.collect(steps, H.replay(model, steps, most), model.vocab_size), refs, dtype)


def test_the_sharing_layers_keep_no_rows_of_their_own(loaded):
    model, *_ = loaded("shared", "float32")
    cache = model.new_cache(640)
    calls = {(g.request.head_dim, g.request.values): g.n_calls for g in cache.kv_groups}
    assert calls == {(16 + 8, False): 1, (24 + 4, False): 1, (8, True): 1}


@pytest.mark.parametrize("name", ["shared", "wide", "mixed"])
def test_greedy_generation_through_the_entry_point(loaded, name):
    """generate(): the scheduler's batches, recorded decode steps, the device's argmax — against the oracle's greedy loop."""
    import llmi_b200 as L
    model, _, _, cfg, w = loaded(name, "float32")
    rng = np.random.default_rng(3)
    prompts = [rng.integers(0, cfg["vocab"], n).tolist() for n in (1, 9, 70, 4, 33)]
    new = [12, 5, 12, 1, 9]
    out = L.generate(model, prompts, max_new=new, max_batch=3)
    ref = [G.generate_greedy(cfg, w, p, n) for p, n in zip(prompts, new)]
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


def test_the_same_steps_again_and_again_give_the_same_bits(loaded):
    """A prompt and eight single tokens of five sequences, six times over on one model: bit for bit."""
    import llmi_b200 as L
    model, _, _, cfg, _ = loaded("wide", "bfloat16")
    rng = np.random.default_rng(1)
    toks = [rng.integers(0, cfg["vocab"], n + 8).tolist() for n in (3, 64, 65, 120, 200)]
    first = None
    for _ in range(6):
        cache = model.new_cache(64 * 20)
        slots = [cache.alloc_slot() for _ in toks]
        out = [model.step(cache, [L.SequenceStep(s, t[:-8], [len(t) - 9]) for s, t in zip(slots, toks)]).cpu().numpy()]
        for j in range(8):
            out.append(model.step(cache, [L.SequenceStep(s, [t[len(t) - 8 + j]], [0]) for s, t in zip(slots, toks)]).cpu().numpy())
        if first is None:
            first = out
        assert all(np.array_equal(a, b) for a, b in zip(first, out))


def test_programs_as_a_user_calls_them(tmp_path):
    """bin/llmi-generate and bin/trace_run on a Sobezen folder, as subprocesses: the design is chosen by config.json."""
    import json
    import os
    import subprocess
    import sys
    from conftest import ROOT
    cfg = M.CONFIGS["mixed"]
    d = str(tmp_path / "model")
    w = M.write_model(d, cfg, M.make_weights(cfg, 7), "F32")
    prompt = [3, 17, 80, 4, 4, 56]
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "llmi-generate"), d, "--ids", ",".join(map(str, prompt)),
                        "--max-new", "6", "--json", "--dtype", "fp32"], capture_output=True, text=True, timeout=200)
    assert r.returncode == 0, r.stderr[-2000:]
    assert json.loads(r.stdout.strip().splitlines()[-1])["generated_ids"] == G.generate_greedy(cfg, w, prompt, 6)
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


# ----------------------------------------------------------------------------- keys that stand out

def far_key_model(kind, at, n, dims):
    """A model of one layer whose logits at the last position show one key and nothing else: token 0 everywhere, token 1 at
    position ``at``, token 2 last.  Token 2's query meets token 1's key with a score of about 30 above all others; the value of
    token 1 moves the logit of id 5, everybody else's that of id 6."""
    W, V = 16, 8
    dim, rot = dims
    if kind == "attention":
        cfg = M.config(W, V, [(M.att(2, 1, dim, rot=rot, scale=1.0), None)], scale=1.0, logit_scale=1.0)
    else:
        cfg = M.config(W, V, [(M.lat(2, dim, rot, 4, dim, 4, scale=1.0), None)], scale=1.0, logit_scale=1.0)
    w = {k: np.zeros_like(v) for k, v in M.make_weights(cfg, 0).items()}
    for k in w:
        if k.endswith("norm1") or k.endswith(".norm") or k.endswith("ls1"):
            w[k][:] = 1.0
    w["embed"][0, 0] = w["embed"][1, 1] = w["embed"][2, 2] = 4.0       # (the norm makes each of them sqrt(W) = 4)
    last = dim - 1                                                      # an entry that no rotation turns
    if kind == "attention":
        w["l0.mix.q"][dim + last, 2] = 2.0                              # the second query head, token 2
        w["l0.mix.k"][last, 1] = 1.0                                    # token 1's key and value
        w["l0.mix.k"][last - 1, 0] = 1.0                                # everybody else's value
        w["l0.mix.o"][3, dim + last], w["l0.mix.o"][4, dim + last - 1] = 1.0, 1.0
    else:
        w["l0.mix.dq"][0, 2] = 1.0
        w["l0.mix.uq"][(dim + rot) + last, 0] = 5.0                     # (a query latent with one entry has size 2)
        w["l0.mix.dkv"][last, 1] = w["l0.mix.dkv"][last - 1, 0] = 1.0
        w["l0.mix.uk"][dim + last, last] = 1.0
        w["l0.mix.uv"][4, last] = w["l0.mix.uv"][5, last - 1] = 1.0
        w["l0.mix.o"][3, 4], w["l0.mix.o"][4, 5] = 1.0, 1.0
    w["head"][5, 3] = w["head"][6, 4] = 1.0
    toks = [0] * n
    toks[at], toks[-1] = 1, 2
    return cfg, w, toks


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("kind,dims", [("attention", (10, 4)), ("attention", (32, 16)), ("attention", (64, 32)), ("attention", (96, 32)),
                                       ("latent_attention", (10, 4)), ("latent_attention", (64, 16))])
def test_one_far_key_in_prompts_and_decoding(kind, dims, dtype, tmp_path):
    """One key among 400, at the first positions, at page borders, just behind and just ahead of the query: whole, decoded, and in
    portions.  The logits say whether it was seen; the token before the last (whose query meets nothing) does not see it."""
    import llmi_b200 as L
    n = 400
    for i, at in enumerate([0, 1, 63, 64, 65, 127, 128, 319, 320, 383, 384, 397, 398]):
        cfg, w, toks = far_key_model(kind, at, n, dims)
        if i == 0:
            weights = M.write_model(str(tmp_path / "m"), cfg, w, STORAGE[dtype])
            model = L.load(str(tmp_path / "m"), dtype)
        ref = G.forward(cfg, weights, toks)
        assert ref[-1, 5] > 1.5 and ref[-1, 6] < 0.1 and ref[-2, 5] < 0.1          # (what the weights were made for)
        for cut in ([n], [n - 1, 1], [n - 40] + [1] * 40, [2, 198, 2, 100, 98], [64, 64, 128, 143, 1]):
            cache = model.new_cache(64 * 8)
            slot, pos = cache.alloc_slot(), 0
            for c in cut:
                out = model.step(cache, [L.SequenceStep(slot, toks[pos:pos + c], [c - 1])])
                pos += c
            got = out.cpu().numpy()[0]
            assert np.abs(got - ref[-1]).max() < (1e-4 if dtype == "float32" else 6e-2), (at, cut[:3], got, ref[-1])


# ----------------------------------------------------------------------------- kernels alone

class _Ctx:
    pass


def _ctx(q_lens, first_pos, slots=None):
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
    ctx.seq_slot = torch.tensor(list(range(len(q_lens))) if slots is None else slots, dtype=torch.int32, device=dev)
    ctx.host_q_lens, ctx.host_kv_lens = list(q_lens), [p + n for p, n in zip(first_pos, q_lens)]
    return ctx


# (tokens, inner, rows): the weight-streaming kernel, the cluster kernel, the single-SM tcgen05 kernel, pairs of SMs, rows
# that nothing aligns
PRODUCTS = [(1, 128, 48), (8, 192, 160), (16, 64, 4096), (30, 128, 96), (60, 256, 2048), (100, 192, 300), (257, 128, 640), (300, 72, 520),
            (700, 256, 4224), (1030, 136, 2560), (5, 50, 22), (300, 50, 22)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,K,N", PRODUCTS)
def test_products_that_scale_what_they_store_or_add(T, K, N, dtype):
    import torch
    from llmi_b200.ops import kernels
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator(device="cuda:0").manual_seed(T + N)
    x = torch.randn(T, K, generator=g, device="cuda:0").to(dt)
    w = (torch.randn(N, K, generator=g, device="cuda:0") * K ** -0.5).to(dt)
    b, s = torch.randn(N, generator=g, device="cuda:0"), 1.0 + torch.randn(N, generator=g, device="cuda:0")
    plain = x.double() @ w.double().T
    for bias, scale in ((b, s), (None, s), (b, None)):
        ref = (plain + (0 if bias is None else bias.double())) * (1 if scale is None else scale.double())
        y0 = torch.randn(T, N, generator=g, device="cuda:0")
        y = y0.clone()
        kernels.linear(x, w, y, bias, kernels.OUT_ADD_F32, oscale=scale)
        assert float((y.double() - (ref + y0.double())).abs().max()) < 2e-5 * float(ref.abs().max() + 1)
        kernels.linear(x, w, y, bias, kernels.OUT_STORE_F32, oscale=scale)
        assert float((y.double() - ref).abs().max()) < 2e-5 * float(ref.abs().max() + 1)
        z = torch.empty(T, N, dtype=dt, device="cuda:0")
        kernels.linear(x, w, z, bias, kernels.OUT_STORE, oscale=scale)
        assert float((z.double() - ref).abs().max()) < (2e-5 if dtype == "float32" else 5e-3) * float(ref.abs().max() + 1)
    kernels.check_device_errors(torch.device("cuda:0"))


def test_a_norm_that_rides_on_a_scaled_product():
    """The residual-adding product that fills the norm behind it fills it from what it has added, factor included."""
    import torch
    from llmi_b200.ops import kernels
    g = torch.Generator(device="cuda:0").manual_seed(0)
    T, K, N = 6, 128, 192
    x = torch.randn(T, K, generator=g, device="cuda:0").bfloat16()
    w, s = (torch.randn(N, K, generator=g, device="cuda:0") * 0.1).bfloat16(), torch.randn(N, generator=g, device="cuda:0")
    nw, y = 1 + 0.3 * torch.randn(N, generator=g, device="cuda:0"), torch.randn(T, N, generator=g, device="cuda:0")
    ref = y.double() + (x.double() @ w.double().T) * s.double()
    then = kernels.DeferredNorm(nw, 1e-5, torch.empty(T, N, dtype=torch.bfloat16, device="cuda:0"),
                                torch.empty((N + 15) // 16, kernels.DeferredNorm.SS_STRIDE, device="cuda:0"))
    assert kernels.linear(x, w, y, None, kernels.OUT_ADD_F32, then, s)
    w2, out = (torch.randn(64, N, generator=g, device="cuda:0") * 0.1).bfloat16(), torch.empty(T, 64, device="cuda:0")
    kernels.linear(then, w2, out, None, kernels.OUT_STORE_F32)
    normed = ref / (ref.pow(2).mean(1, keepdim=True) + 1e-5).sqrt() * nw.double()
    assert float((out.double() - normed @ w2.double().T).abs().max()) < 2e-2 and float((y.double() - ref).abs().max()) < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("T,K,F", [(1, 128, 24), (8, 192, 80), (16, 64, 2048), (30, 128, 48), (60, 256, 1024), (100, 192, 150), (257, 128, 320),
                                   (300, 72, 260), (700, 256, 2112), (1030, 136, 1280), (5, 50, 11), (130, 50, 11)])
def test_bounded_gate_on_every_product(T, K, F, dtype):
    """Gate and up values on both sides of both bounds, with biases; the product that gates in its epilogue and the two steps."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.parts.registry import get_part
    from llmi_b200.parts.spec import PartSpec
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    g = torch.Generator().manual_seed(T + F)
    W, limit, alpha = K, 1.25, 1.702
    t = {"gate": torch.randn(F, K, generator=g) * 2 * K ** -0.5, "gate.b": torch.randn(F, generator=g), "up": torch.randn(F, K, generator=g) * 2 * K ** -0.5,
         "up.b": torch.randn(F, generator=g), "down": torch.randn(W, F, generator=g) * F ** -0.5, "down.b": torch.randn(W, generator=g)}
    t = {k: v.to(dt) for k, v in t.items()}
    rt = Runtime(dt, "cuda:0")
    spec = PartSpec("swiglu", {"width": W, "inner": F, "activation": "bounded", "alpha": alpha, "limit": limit, "bias": True, "names": ("gate", "up", "down")})
    ff = get_part("ffn", "swiglu")(spec, t, rt)
    x = torch.randn(T, K, generator=g).to(dt).to("cuda:0")
    y, s = torch.zeros(T, W, device="cuda:0"), torch.randn(W, generator=g).to("cuda:0")
    ff.forward(x, y, None, out_scale=s)
    n = {k: v.double().numpy() for k, v in t.items()}
    xn = x.double().cpu().numpy()
    z, u = xn @ n["gate"].T + n["gate.b"], xn @ n["up"].T + n["up.b"]
    for v in (z, u):
        assert (v > limit).any() and (v < -limit).any()
    ref = (G.bounded_gate(z, u, limit) @ n["down"].T + n["down.b"]) * s.double().cpu().numpy()
    err = np.abs(y.cpu().numpy() - ref).max() / np.abs(ref).max()
    assert err < (1e-5 if dtype == "float32" else 1.5e-2), err


def _delta_inputs(T, dims, ranks, seed, keep=False):
    H_, Hk, D, Dv, K = dims
    rng = np.random.default_rng(seed)
    n_conv = 2 * Hk * D + H_ * Dv
    proj = rng.standard_normal((T, n_conv + H_ + sum(ranks) + 3)).astype(np.float32)
    conv = (rng.standard_normal((n_conv, K)) / np.sqrt(K)).astype(np.float32)
    a_log = (np.full(H_, -9.0) if keep else np.log(rng.uniform(0.05, 1.5, H_))).astype(np.float32)
    dt_bias = rng.standard_normal(H_ * D).astype(np.float32)
    w2 = [(rng.standard_normal((n, r)) / np.sqrt(r)).astype(np.float32) for n, r in ((H_ * D, ranks[0]), (H_ * Dv, ranks[1]))]
    norm = (1 + 0.2 * rng.standard_normal(Dv)).astype(np.float32)
    return proj, conv, a_log, dt_bias, w2, norm


def _delta_reference(proj, conv, a_log, dt_bias, w2, norm, dims, ranks, eps):
    """One sequence from its start: o [T, H*Dv] behind the norm and the gate."""
    H_, Hk, D, Dv, K = dims
    T, x = proj.shape[0], proj.astype(np.float64)
    n_qk, n_conv = Hk * D, 2 * Hk * D + H_ * Dv
    y = G.silu(G.short_conv(x[:, :n_conv], conv.astype(np.float64)))
    q, k, v = y[:, :n_qk].reshape(T, Hk, D), y[:, n_qk:2 * n_qk].reshape(T, Hk, D), y[:, 2 * n_qk:].reshape(T, H_, Dv)
    unit = lambda a: a / np.sqrt(np.sum(a * a, axis=-1, keepdims=True) + 1e-6)      # noqa: E731
    of = np.arange(H_) // (H_ // Hk)
    at = n_conv + H_
    low_a, low_g = x[:, at:at + ranks[0]], x[:, at + ranks[0]:at + sum(ranks)]
    g = np.exp(-np.exp(a_log.astype(np.float64))[None, :, None] * G.softplus(low_a @ w2[0].T + dt_bias).reshape(T, H_, D))
    o = G.delta_walk(unit(q)[:, of] * D ** -0.5, unit(k)[:, of], v, G.logistic(x[:, n_conv:n_conv + H_]), g)
    return (G.rms(o, eps) * norm * G.logistic(low_g @ w2[1].T).reshape(T, H_, Dv)).reshape(T, -1)


DELTA_SIZES = [(2, 1, 8, 8, 3), (4, 2, 32, 48, 4), (2, 2, 64, 64, 2), (3, 1, 128, 96, 4), (2, 2, 128, 128, 1), (6, 3, 96, 40, 3), (1, 1, 256, 256, 2),
               (2, 1, 4, 200, 5), (3, 3, 10, 7, 2), (2, 2, 32, 16, 16), (2, 1, 72, 132, 4)]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dims", DELTA_SIZES)
def test_delta_rule_kernels_with_a_decay_per_channel(dims, dtype):
    """Three sequences on slots out of order, one of them without a slot: prompts of unequal lengths by the general kernels, then
    single tokens by their own (where the sizes are theirs) and by the general ones — the same outputs and the same state."""
    import torch
    from llmi_b200.ops import kernels
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    H_, Hk, D, Dv, K = dims
    ranks, eps, n_single = (5, 12), 1e-5, 6
    lens, slots = [9, 1, 20], [3, 1, 0]
    dev = lambda a: torch.tensor(np.ascontiguousarray(a), device="cuda:0")        # noqa: E731
    one = [_delta_inputs(n + n_single, dims, ranks, 11, keep=True) for n in lens]
    conv, a_log, dt_bias, w2, norm = one[0][1:]
    rng = np.random.default_rng(5)
    projs = [rng.standard_normal(p[0].shape).astype(np.float32) for p in one]
    refs = [_delta_reference(p, conv, a_log, dt_bias, w2, norm, dims, ranks, eps) for p in projs]
    n_conv = 2 * Hk * D + H_ * Dv
    n_state = kernels.delta_state_floats(*dims)
    state = torch.full((5, n_state), float("nan"), device="cuda:0")
    for s in slots:
        state[s].zero_()
    at, n_prep = n_conv + H_, n_conv + H_ * D + H_
    n_prep += -n_prep % 4
    t_conv, t_alog, t_dtb, t_norm = dev(conv), dev(a_log), dev(dt_bias), dev(norm)

    def general(proj, ctx, st):
        T = proj.shape[0]
        z = proj[:, at:at + ranks[0]].double() @ dev(w2[0]).double().T
        gate = (proj[:, at + ranks[0]:at + sum(ranks)].double() @ dev(w2[1]).double().T).float()
        prep = torch.full((T, n_prep), float("nan"), device="cuda:0")
        o, out = torch.full((T, H_ * Dv), float("nan"), device="cuda:0"), torch.full((T, H_ * Dv), float("nan"), dtype=dt, device="cuda:0")
        kernels.delta_step(proj, dims, t_conv, t_alog, t_dtb, st, ctx, prep, o, z=z.float())
        kernels.delta_finish(o, gate, t_norm, eps, H_, Dv, ctx, out, kernels.GATE_SIGMOID)
        return out.float().cpu().numpy()

    tol = 3e-5 if dtype == "float32" else 2e-2
    scale = max(1.0, max(np.abs(r).max() for r in refs))
    got = general(dev(np.concatenate([p[:n] for p, n in zip(projs, lens)])), _ctx(lens, [0, 0, 0], slots), state)
    want = np.concatenate([r[:n] for r, n in zip(refs, lens)])
    assert np.abs(got - want).max() < tol * scale, float(np.abs(got - want).max())
    assert bool(torch.isnan(state[2]).all()) and bool(torch.isnan(state[4]).all())
    # single tokens: a padding row of no sequence in the middle
    single = kernels.channel_token_supported(dims, *ranks) and n_state % 4 == 0
    assert single == (D % 4 == 0 and Dv % 4 == 0)
    pad = lambda a: torch.nn.functional.pad(dev(a.T), (0, -a.shape[0] % 64)).to(dt).contiguous()         # noqa: E731
    other = state.clone()
    for j in range(n_single):
        rows = [p[n + j] for p, n in zip(projs, lens)]
        ctx = _ctx([1, 1, 1, 1], [lens[0] + j, 0, lens[1] + j, lens[2] + j], [slots[0], -1, slots[1], slots[2]])
        ctx.tok_seq[1] = -1
        proj = dev(np.stack([rows[0], np.full_like(rows[0], np.nan), rows[1], rows[2]]))
        want = np.stack([r[n + j] for r, n in zip(refs, lens)])
        got = general(proj, ctx, other)
        assert np.abs(got[[0, 2, 3]] - want).max() < tol * scale and (got[1] == 0).all()
        if single:
            prep = torch.full((4, n_prep), float("nan"), device="cuda:0")
            gate = torch.full((4, H_ * Dv), float("nan"), device="cuda:0")
            out = torch.full((4, H_ * Dv), float("nan"), dtype=dt, device="cuda:0")
            kernels.channel_token(proj, dims, (at, ranks[0]), (at + ranks[0], ranks[1]), t_conv, t_alog, t_dtb, pad(w2[0]), pad(w2[1]), state, ctx,
                                  prep, gate, t_norm, eps, out)
            mine = out.float().cpu().numpy()
            assert np.abs(mine[[0, 2, 3]] - want).max() < tol * scale and (mine[1] == 0).all(), float(np.abs(mine[[0, 2, 3]] - want).max())
            for s in slots:
                assert float((state[s] - other[s]).abs().max()) < (1e-4 if dtype == "float32" else 2e-2)
            assert bool(torch.isnan(state[2]).all()) and bool(torch.isnan(state[4]).all())


def test_a_state_that_is_not_to_be_written_stays():
    import torch
    from llmi_b200.ops import kernels
    dims, ranks = (2, 1, 32, 64, 3), (4, 4)
    proj, conv, a_log, dt_bias, w2, norm = _delta_inputs(2, dims, ranks, 3)
    dev = lambda a: torch.tensor(np.ascontiguousarray(a), device="cuda:0")        # noqa: E731
    state = torch.randn(3, kernels.delta_state_floats(*dims), device="cuda:0")
    before, at = state.clone(), 2 * 32 + 2 * 64 + 2
    out, prep = torch.empty(2, 128, device="cuda:0"), torch.empty(2, at + 64 + 2, device="cuda:0")
    pad = lambda a: torch.nn.functional.pad(dev(a.T), (0, -a.shape[0] % 64)).contiguous()                 # noqa: E731
    kernels.channel_token(dev(proj), dims, (at, 4), (at + 4, 4), dev(conv), dev(a_log), dev(dt_bias), pad(w2[0]), pad(w2[1]), state, _ctx([1, 1], [5, 9]),
                          prep, torch.empty(2, 128, device="cuda:0"), dev(norm), 1e-5, out, write_state=False)
    assert torch.equal(state, before) and bool(torch.isfinite(out).all())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("Hq,D,C,R,Q", [(3, 8, 24, 8, 12), (2, 16, 64, 32, 64), (5, 6, 9, 2, 7)])
def test_latent_rows_and_queries_with_stretched_angles(Hq, D, C, R, Q, dtype):
    """The preparation of a latent layer with a rotation that also scales: cache rows, query latent, rotated queries; and, for a
    layer that reads another one's rows, nothing but the query latent."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.ops import kernels
    from llmi_b200.parts.registry import get_part
    from llmi_b200.parts.spec import PartSpec
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(C)
    lens, starts, page, eps = [5, 8], [60, 0], 64, 1e-4
    T = sum(lens)
    rot = {"base": 700.0, "dims": R, "scaling": {"factor": 6.0, "original": 50.0, "fast": 6.0, "slow": 0.5}}
    part = get_part("position", "rotary_pairs")(PartSpec("rotary_pairs", {"head_dim": R, "rotary_dim": R, "theta": 700.0, "scaling": rot["scaling"]}), {},
                                               Runtime(dt, "cuda:0"))
    f, amp = G.frequencies(rot)
    assert np.allclose(part.inv_freq.cpu().numpy(), f, rtol=1e-6) and math.isclose(part.amplitude, amp) and amp > 1
    down = rng.standard_normal((T, Q + C + R)).astype(np.float32)
    wq, wc = ((1 + 0.3 * rng.standard_normal(n)).astype(np.float32) for n in (Q, C))
    ctx = _ctx(lens, starts)
    pos = ctx.tok_pos.cpu().numpy()
    pages = torch.tensor([[2, 4], [1, -1]], dtype=torch.int32, device="cuda:0")
    cache = torch.full((5, 1, page, C + R), float("nan"), dtype=dt, device="cuda:0")
    cq = torch.full((T, Q), float("nan"), dtype=dt, device="cuda:0")
    dev = lambda a: torch.tensor(np.ascontiguousarray(a), device="cuda:0")        # noqa: E731
    kernels.latent_prepare(dev(down[:, :Q]), Q, C, R, dev(wq), None, eps, part.inv_freq, R, ctx, pages, page, cache, cq, write_kv=False,
                           amplitude=part.amplitude)
    assert bool(torch.isnan(cache).all())
    x = down.astype(np.float64)
    ref_q = G.rms(x[:, :Q], eps) * wq
    tol = 2e-5 if dtype == "float32" else 3e-2
    assert np.abs(cq.float().cpu().numpy() - ref_q).max() < tol
    cq.fill_(float("nan"))
    kernels.latent_prepare(dev(down), Q, C, R, dev(wq), dev(wc), eps, part.inv_freq, R, ctx, pages, page, cache, cq, amplitude=part.amplitude)
    assert np.abs(cq.float().cpu().numpy() - ref_q).max() < tol

    def turn(v, p):
        return G.rotate(np.broadcast_to(v, (int(p) + 1, *v.shape)), rot)[-1]
    c = G.rms(x[:, Q:Q + C], eps) * wc
    q = rng.standard_normal((T, Hq * (D + R))).astype(np.float32)
    tq = torch.tensor(q, device="cuda:0").to(dt)
    qa = torch.full((T, Hq * (C + R)), float("nan"), dtype=dt, device="cuda:0")
    kernels.latent_q_rotate(tq, D, qa, C, R, Hq, part.inv_freq, R, ctx, 1, part.amplitude)
    got, q64 = qa.float().cpu().numpy().reshape(T, Hq, C + R), tq.double().cpu().numpy().reshape(T, Hq, D + R)
    assert np.isnan(got[..., :C]).all()
    for t in range(T):
        row = cache[int(pages[0 if t < lens[0] else 1, pos[t] // page]), 0, pos[t] % page].float().cpu().numpy()
        assert np.abs(row[:C] - c[t]).max() < tol and np.abs(row[C:] - turn(x[t, Q + C:], pos[t])).max() < tol
        assert np.abs(got[t, :, C:] - turn(q64[t, :, D:], pos[t])).max() < tol
    assert int((~torch.isnan(cache)).sum()) == T * (C + R)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("sizes", [(4, 2, 48), (2, 1, 96), (8, 8, 64), (6, 3, 128), (5, 5, 10), (16, 1, 80), (32, 1, 16)])
def test_keys_as_values_over_pages_out_of_order(sizes, dtype):
    """300 positions on pages that are not in order, everything else NaN: keys rotated, values as projected, from the product's
    rows with their biases; the queries of a single token and of portions of 70 and 200."""
    import torch
    from llmi_b200.engine.runtime import Runtime
    from llmi_b200.ops import kernels
    Hq, Gk, D = sizes
    dt = {"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype]
    rng = np.random.default_rng(D)
    N, page, scale, dims = 300, 64, 1.2 * D ** -0.5, D // 4 * 2
    proj = torch.tensor(rng.standard_normal((N, (Hq + Gk) * D)).astype(np.float32), device="cuda:0")
    rot = {"base": 500.0, "dims": dims}
    f = torch.tensor(G.frequencies(rot)[0].astype(np.float32), device="cuda:0")
    order = rng.permutation(9)[:5]
    pages = torch.tensor(order[None, :].astype(np.int32), device="cuda:0")
    x = proj.double().cpu().numpy()
    q, v = G.rotate(x[:, :Hq * D].reshape(N, Hq, D), rot), x[:, Hq * D:].reshape(N, Gk, D)
    k = G.rotate(v, rot)
    rt = Runtime(dt, "cuda:0")
    ref = np.zeros((N, Hq, D))
    for h in range(Hq):
        s = q[:, h] @ k[:, h // (Hq // Gk)].T * scale
        ref[:, h] = G.softmax(np.where(np.tril(np.ones((N, N), bool)), s, -np.inf)) @ v[:, h // (Hq // Gk)]
    for n_rows in (1, 70, 200):
        kc, vc = (torch.full((10, Gk, page, D), float("nan"), dtype=dt, device="cuda:0") for _ in range(2))
        for lo, hi in ((0, N - n_rows), (N - n_rows, N)):
            ctx = _ctx([hi - lo], [lo])
            qo = torch.full((hi - lo, Hq * D), float("nan"), dtype=dt, device="cuda:0")
            kernels.qkv_prepare(proj[lo:hi], Hq, Gk, D, Gk, D, None, None, 0.0, f, dims, ctx, pages, page, kc, vc, qo, pairing=1, v_from_k=True)
        out = torch.full((n_rows, Hq * D), float("nan"), dtype=dt, device="cuda:0")
        kernels.attention_maps(qo, out, kc, vc, ctx, pages, page, Hq, Gk, 1, D, D, scale, None, 0, 0, rt=rt)
        kernels.check_device_errors(torch.device("cuda:0"))
        got = out.float().cpu().numpy().reshape(n_rows, Hq, D)
        assert np.isfinite(got).all() and np.abs(got - ref[N - n_rows:]).max() < (2e-5 if dtype == "float32" else 4e-2)
