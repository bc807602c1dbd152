"""Nurinex on the GPU against the plain numpy oracle, in f32 (tight) and in bf16 (the precision it is served in):
each mechanism with its absence ruled out, prompts, decoding, portions, reused caches, far keys, edges, scoring and
generation through the serving front."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from ferrum_cpu_b200 import FerrumCudaError, _lib, decoder, engine, registry
from ferrum_cpu_b200.backend import CudaBackend, GenRequest
from ferrum_cpu_b200.decoder import CudaNurinex
from tests.nurinex_models import MD, NO, L, build, configs, error, ids, needle

pytestmark = pytest.mark.gpu
F32, BF16 = _lib.FC_MATH_FP32, _lib.FC_MATH_BF16
TOL = {F32: 2e-5, BF16: 2.5e-2}
MODES = pytest.mark.parametrize("mode", [F32, BF16], ids=["f32", "bf16"])


def feed_in(model, cache, toks, cuts):
    """Logits of every token, fed in portions that end at `cuts`."""
    out, at = np.empty((len(toks), model.info.vocab), dtype=np.float32), 0
    for e in list(cuts) + [len(toks)]:
        if e > at:
            out[at:e] = model.feed(toks[at:e], cache, range(e - at))
            at = e
    return out


def check(path, config, ten, mode, toks, cuts=(), want=None, ctx=None):
    want = NO.forward(config, ten, toks) if want is None else want
    m = CudaNurinex(path, math_mode=mode, ctx=ctx or len(toks))
    got = feed_in(m, m.new_cache(), toks, cuts)
    m.close()
    assert error(got, want) < TOL[mode], error(got, want)
    return got, want


# ------------------------------------------------------------------------------- whole models
@MODES
@pytest.mark.parametrize("name", sorted(configs()))
def test_prompt_decode_and_portions_match_the_oracle(tmp_path, name, mode):
    config, rows, rank = configs()[name]
    path, ten = build(tmp_path, config, 5, rows, rank)
    toks = ids(2, 150, config["vocab"])
    want = NO.forward(config, ten, toks)
    m = CudaNurinex(path, math_mode=mode, ctx=160)
    c = m.new_cache()
    for cuts in ([], range(1, 150), [2, 4, 7, 12, 29, 31, 64, 66, 67, 128], [100] + list(range(101, 150)), range(2, 150, 2)):
        c.clear()
        got = feed_in(m, c, toks, cuts)
        assert c.pos() == 150
        assert error(got, want) < TOL[mode], (list(cuts)[:4], error(got, want))
    m.close()


@MODES
def test_residual_stream_after_every_layer(tmp_path, mode):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 6, rows, rank)
    toks = ids(3, 40, config["vocab"])
    lay = []
    NO.forward(config, ten, toks, lay)
    m = CudaNurinex(path, math_mode=mode, ctx=64)
    c = m.new_cache()
    got = np.concatenate([m.feed_layers(toks[:23], c), m.feed_layers(toks[23:], c)], axis=1)
    for i, w in enumerate(lay):
        assert np.abs(got[i] - w).max() < (2e-6 if mode == F32 else 2e-2) * np.abs(w).max(), i
    m.close()


@MODES
def test_portions_do_not_change_the_logits(tmp_path, mode):
    """Beyond rounding the cut does not matter: not in portions, nor token by token."""
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 7, rows, rank)
    toks = ids(4, 300, config["vocab"])
    m = CudaNurinex(path, math_mode=mode, ctx=300)
    c = m.new_cache()
    whole = feed_in(m, c, toks, [])
    for cuts in ([128], [63, 65, 191], [2, 298], [7 * k for k in range(1, 42)]):
        c.clear()
        got = feed_in(m, c, toks, cuts)
        assert error(got, whole) < TOL[mode] / 4, cuts
    c.clear()
    got = feed_in(m, c, toks, range(250, 300))
    assert error(got, whole) < TOL[mode]
    m.close()


# --------------------------------------------------------------------- one mechanism at a time
def one_layer(**kw):
    return MD.nurinex_config(180, 64, [L(heads=6, kv_heads=2, dim=32, vdim=24, bias_max=60, coef=0.6, every=10, r_heads=2, r_dim=32, ff=80, **kw)],
                             eps=1e-2, emb_scale=2.5)


def only(side):
    """Weights that leave one of the three sublayers."""
    def edit(ten):
        if side != "left":
            ten["l0.mix.left.out"][:] = 0
        if side != "right":
            ten["l0.mix.right.out"][:] = 0
        if side != "ff":
            ten["l0.mlp.down"][:] = 0
    return edit


MECHANISMS = {
    # name: (sublayer that is left, the oracle without the mechanism as (function, replacement))
    "sink": ("left", ("softmax_with_sink", lambda s, k: np.exp(s - s.max()) / np.exp(s - s.max()).sum())),
    "query temperature": ("left", ("query_temperature", lambda p, c, e: 1.0)),
    "temperature one token early": ("left", ("query_temperature", lambda p, c, e: 1 + c * np.log((p + 2) // e + 1))),
    "bias of the distance": ("left", ("distance_bucket", lambda n, rows, far: 0)),
    "bias buckets one off": ("left", ("distance_bucket", lambda n, rows, far, f=NO.distance_bucket: f(n + 1, rows, far))),
    "decay": ("right", ("decay", lambda m, w: np.ones((m.shape[0], w["w0"].size)))),
    "token shift": ("right", ("token_shift", lambda h: h)),
    "gate": ("right", ("silu", lambda z: z)),
    "activation": ("ff", ("xielu", lambda z, p, q: np.maximum(z, 0) ** 2)),
}


@MODES
@pytest.mark.parametrize("what", sorted(MECHANISMS))
def test_each_mechanism_shows(tmp_path, monkeypatch, what, mode):
    side, (fn, without) = MECHANISMS[what]
    config = one_layer()
    path, ten = build(tmp_path, config, 8, 8, 6, only(side))
    toks = ids(5, 90, config["vocab"])
    for cuts in ([], range(30, 90)):
        got, _ = check(path, config, ten, mode, toks, cuts)
    monkeypatch.setattr(NO, fn, without)
    assert error(got, NO.forward(config, ten, toks)) > 2 * TOL[mode]       # an oracle without it is told apart


WEIGHTS_THAT_COUNT = ["l0.norm1", "l0.mix.left.talk", "l0.mix.left.rel", "l0.mix.left.sink", "l0.mix.left.out", "l0.mix.right.out",
                      "l0.mix.right.mu.r", "l0.mix.right.mu.k", "l0.mix.right.mu.v", "l0.mix.right.mu.g", "l0.mix.right.mu.w",
                      "l0.mix.right.u", "l0.mix.right.norm", "l0.mix.right.w0", "l0.mix.right.w1", "l0.mix.right.w2", "l0.mlp.act",
                      "final.norm"]


def test_every_small_tensor_reaches_the_result(tmp_path):
    """f32: matches the oracle, and an oracle with that tensor's entries turned round does not match."""
    config = one_layer()
    toks = ids(6, 60, config["vocab"])
    path, ten = build(tmp_path, config, 9, 8, 6)
    got, _ = check(path, config, ten, F32, toks)
    for name in WEIGHTS_THAT_COUNT:
        changed = dict(ten, **{name: np.ascontiguousarray(ten[name].ravel()[::-1].reshape(ten[name].shape))})
        assert error(got, NO.forward(config, changed, toks)) > 50 * TOL[F32], name


def test_constants_are_read_from_the_configuration(tmp_path):
    toks = ids(7, 70, 180)
    base = one_layer()

    def variant(**left):
        c = copy.deepcopy(base)
        c["layers"][0]["mixer"]["left"].update(left)
        return c
    cases = [base, variant(scale=0.05), variant(bias_max=31), variant(q_temp={"coef": -0.3, "every": 3}), variant(q_temp={"coef": 0.4, "every": 2.5}),
             dict(base, norm={"eps": 1e-6}), dict(base, embedding={"scale": 0.5})]
    _, ten = build(tmp_path / "w", base, 10, 8, 6)
    results = []
    for i, c in enumerate(cases):
        p = MD.write(str(tmp_path / str(i)), c, {n: MD.to_bf16(a).reshape(a.shape) for n, a in ten.items()})
        results.append(check(p, c, ten, F32, toks, range(40, 70))[0])
    for i in range(1, len(cases)):
        assert error(results[i], results[0]) > 20 * TOL[F32], i


@MODES
def test_activation_on_both_sides_and_far_out(tmp_path, mode):
    config = one_layer()

    def edit(ten):
        only("ff")(ten)
        ten["l0.mlp.up"] *= 6                       # arguments from about -15 to 15
    path, ten = build(tmp_path, config, 11, 8, 6, edit)
    check(path, config, ten, mode, ids(8, 50, config["vocab"]), range(25, 50))


@MODES
def test_decays_from_forgetting_at_once_to_never(tmp_path, mode):
    config = one_layer()

    def edit(ten):
        only("right")(ten)
        n = ten["l0.mix.right.w0"].size
        ten["l0.mix.right.w0"] = np.linspace(-14.0, 4.0, n).astype(np.float32)
    path, ten = build(tmp_path, config, 12, 8, 6, edit)
    check(path, config, ten, mode, ids(9, 200, config["vocab"]), [90, 91] + list(range(150, 200)))


# ------------------------------------------------------------------ far keys, edges, first tokens
@MODES
def test_a_far_key_is_found_at_every_distance(tmp_path, mode):
    """One token attends to another one far back; distances sit on tile, split and bucket edges."""
    base = one_layer()
    asks, holds, T, first = 7, 11, 420, 5
    path, ten = build(tmp_path, base, 13, 8, 6, lambda t: (only("left")(t), needle(t, base, asks, holds)))
    toks = ids(10, T, base["vocab"])
    toks[(toks == asks) | (toks == holds)] = 8
    toks[first] = holds
    # 31/32/33, 59..61 (the bias table's end), 63..65, 127..129, 255..257 keys away and more
    later = sorted({first + n for n in (1, 3, 4, 31, 32, 33, 59, 60, 61, 63, 64, 65, 127, 128, 129, 255, 256, 257, 400)})
    for p in later:
        a = toks.copy()
        a[p] = asks
        a = a[:p + 3]
        want = NO.forward(base, ten, a)
        b = a.copy()
        b[first] = 9
        assert error(want[p:p + 1], NO.forward(base, ten, b)[p:p + 1]) > 3 * TOL[mode], p      # the far key matters
        m = CudaNurinex(path, math_mode=mode, ctx=T)
        for cuts in ([], [p], [p, p + 1]):
            got = feed_in(m, m.new_cache(), a, cuts)
            assert error(got[p:p + 1], want[p:p + 1]) < TOL[mode], (p, cuts)
        m.close()


@MODES
def test_first_tokens_and_single_token_sequences(tmp_path, mode):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 14, rows, rank)
    m = CudaNurinex(path, math_mode=mode, ctx=8)
    c = m.new_cache()
    for n in (1, 2, 3, 5):
        toks = ids(20 + n, n, config["vocab"])
        want = NO.forward(config, ten, toks)
        for cuts in ([], [1], range(1, n)):
            c.clear()
            assert error(feed_in(m, c, toks, cuts), want) < TOL[mode]
    m.close()


@MODES
def test_long_decoding(tmp_path, mode):
    """Past many attention splits and temperature steps, token by token from a short prompt."""
    config = one_layer()
    path, ten = build(tmp_path, config, 15, 8, 6)
    toks = ids(11, 700, config["vocab"])
    check(path, config, ten, mode, toks, range(3, 700), ctx=4500)


# ------------------------------------------------------------------------ caches, reuse, refusals
@MODES
def test_caches_are_independent_and_reusable(tmp_path, mode):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 16, rows, rank)
    m = CudaNurinex(path, math_mode=mode, ctx=130)
    seqs = [ids(30 + i, n, config["vocab"]) for i, n in enumerate((130, 3, 57))]
    alone = []
    c = m.new_cache()
    for s in seqs:                                   # one cache for all, longest first: what it held must not show
        c.clear()
        alone.append(feed_in(m, c, s, []))
        assert error(alone[-1], NO.forward(config, ten, s)) < TOL[mode]
    caches = [m.new_cache() for _ in seqs]
    at, got = [0] * 3, [[], [], []]
    rng = np.random.default_rng(0)
    while any(a < len(s) for a, s in zip(at, seqs)):
        i = int(rng.integers(0, 3))
        n = min(int(rng.integers(1, 20)), len(seqs[i]) - at[i])
        if n:
            got[i].append(m.feed(seqs[i][at[i]:at[i] + n], caches[i], range(n)))
            at[i] += n
    for g, a in zip(got, alone):
        assert error(np.concatenate(g), a) < TOL[mode]
    caches[1].close()                                # freed, and another one in its place
    again = m.new_cache()
    assert np.array_equal(feed_in(m, again, seqs[2], []), alone[2])
    m.close()


def test_refusals_leave_the_cache_usable(tmp_path):
    config, rows, rank = configs()["odd"]
    path, ten = build(tmp_path, config, 17, rows, rank)
    m = CudaNurinex(path, math_mode=F32, ctx=20)
    c = m.new_cache()
    toks = ids(12, 20, config["vocab"])
    m.feed(toks[:10], c)
    for bad in ([config["vocab"]], [-1, 3], np.zeros(11, np.int32)):
        with pytest.raises(FerrumCudaError) as e:
            m.feed(bad, c)
        assert e.value.code == _lib.FC_E_DIM and c.pos() == 10
    with pytest.raises(FerrumCudaError):
        m.feed([1, 2], c, [2])
    got = m.feed(toks[10:], c, range(9, -1, -1))[::-1]     # places in any order
    assert error(got, NO.forward(config, ten, toks)[10:]) < TOL[F32]
    with pytest.raises(FerrumCudaError):
        m.feed([1], c)                                     # full
    m.close()


def test_wide_rows_in_portions_of_every_size_class(tmp_path):
    """Rows of 4096 values: the row kernel's staging passes 48 KB in one of the size classes and not in the next."""
    config = MD.nurinex_config(40, 4096, [L(heads=2, kv_heads=1, dim=16, vdim=16, bias_max=50, r_heads=1, r_dim=16, ff=32)])
    path, ten = build(tmp_path, config, 26, 8, 4)
    toks = ids(27, 600, 40)
    m = CudaNurinex(path, math_mode=F32, ctx=600)
    c = m.new_cache()
    whole = feed_in(m, c, toks, [])
    for cuts in ([300], [100, 101], range(560, 600)):
        c.clear()
        assert error(feed_in(m, c, toks, cuts), whole) < TOL[F32]
    assert error(whole[:40], NO.forward(config, ten, toks[:40])) < TOL[F32]
    m.close()


def test_portions_longer_than_one_pass(tmp_path):
    """More tokens than a forward pass takes are cut inside the call; nothing shows at the seam."""
    config = MD.nurinex_config(90, 32, [L(heads=2, kv_heads=1, dim=16, vdim=16, bias_max=500, r_heads=1, r_dim=16, ff=32)])
    path, _ = build(tmp_path, config, 18, 16, 4)
    toks = ids(13, 2300, 90)
    m = CudaNurinex(path, math_mode=F32, ctx=2300)
    c = m.new_cache()
    a = m.feed(toks, c, [0, 2046, 2047, 2048, 2049, 2299])
    c.clear()
    m.feed(toks[:1000], c)
    b = m.feed(toks[1000:], c, [1046, 1047, 1048, 1049, 1299])
    assert error(b, a[1:]) < TOL[F32] / 4
    m.close()


def test_waits_that_run_out_are_reported(tmp_path):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 19, rows, rank)
    m = CudaNurinex(path, math_mode=BF16, ctx=64)
    c = m.new_cache()
    toks = ids(14, 40, config["vocab"])
    _lib.check(_lib.lib().fc_debug_set_wait_budget(200_000, 1))
    try:
        with pytest.raises(FerrumCudaError) as e:
            m.feed(toks, c, [0])
        assert e.value.code == _lib.FC_E_TIMEOUT
    finally:
        _lib.check(_lib.lib().fc_debug_set_wait_budget(4_000_000_000, 0))
    c.clear()
    assert error(feed_in(m, c, toks, []), NO.forward(config, ten, toks)) < TOL[BF16]
    m.close()


# ------------------------------------------------------------------------- scoring and generation
@MODES
def test_scoring_matches_the_oracle(tmp_path, mode):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 21, rows, rank)
    be = CudaBackend(registry.load(path, math_mode=mode, ctx=200))
    toks = ids(15, 120, config["vocab"])
    z = NO.forward(config, ten, toks)
    lp = z - z.max(axis=1, keepdims=True)
    lp = lp - np.log(np.exp(lp).sum(axis=1, keepdims=True))
    per = lp[np.arange(119), toks[1:]]
    tol = 1e-4 if mode == F32 else 0.1
    sc, got, greedy = be.model.score_from(toks, 1, per_token=True)
    assert sc.n_tokens == 119 and np.abs(got - per).max() < tol
    sure = np.sort(z[:-1], axis=1)
    sure = sure[:, -1] - sure[:, -2] > tol
    assert np.array_equal(greedy[sure], (z[:-1].argmax(axis=1) == toks[1:])[sure])
    t1 = be.submit_score(toks[:70], toks[70:])
    t2 = be.submit_score_rolling(toks[:33])
    out = be.flush()
    assert out[t1]["n_tokens"] == 50 and abs(out[t1]["logprob"] - per[69:].sum()) < tol * 50
    assert out[t2]["n_tokens"] == 32 and abs(out[t2]["logprob"] - per[:32].sum()) < tol * 32
    be.model.close()


def test_greedy_generation_through_the_backend(tmp_path):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path, config, 22, rows, rank)
    be = CudaBackend(registry.load(path, math_mode=F32, ctx=128))
    prompt = ids(16, 19, config["vocab"]).tolist()
    seq, margins = list(prompt), []
    for _ in range(30):
        z = NO.forward(config, ten, seq)[-1]
        top = np.sort(z)
        margins.append(top[-1] - top[-2])
        seq.append(int(z.argmax()))
    assert min(margins) > 1e-4
    want = seq[19:]
    for n in (1, 30):
        assert be.generate(GenRequest(prompt, max_tokens=n, temperature=0.0))["tokens"] == want[:n]
    eos = want[12]
    stop = want.index(eos)
    assert be.generate(GenRequest(prompt, max_tokens=30, temperature=0.0, eos=eos))["tokens"] == want[:stop]
    one = be.generate(GenRequest(prompt[:1], max_tokens=5, temperature=0.0))["tokens"]      # a one-token prompt
    seq = prompt[:1]
    for _ in range(5):
        seq.append(int(NO.forward(config, ten, seq)[-1].argmax()))
    assert one == seq[1:]
    long = be.generate(GenRequest(prompt, max_tokens=500, temperature=0.0))["tokens"]       # ends with the context
    assert len(long) == 128 - 19 and long[:30] == want
    # sampling: the same generator state gives the same tokens, and a cancelled request gives none
    req = GenRequest(prompt, max_tokens=20, temperature=0.9, top_k=20, seed=3)
    assert be.generate(req) == be.generate(req)
    assert all(0 <= t < config["vocab"] for t in be.generate(req)["tokens"])
    assert be.generate(GenRequest(prompt, cancel=np.ones(1, np.int32))) is None
    be.model.close()


def test_sampling_with_penalty_equals_the_sampler_on_the_logits(tmp_path):
    config, rows, rank = configs()["odd"]
    path, ten = build(tmp_path, config, 23, rows, rank)
    m = CudaNurinex(path, math_mode=F32, ctx=64)
    prompt = ids(17, 9, config["vocab"])
    params = engine.sampling(temperature=0.7, top_k=0, top_p=0.9, repetition_penalty=1.3)
    got, state = m.generate(prompt, 12, params, rng_state=12345)
    c, seq, st = m.new_cache(), list(prompt), 12345
    z = m.feed(prompt, c, [8])[0]
    for t in got:
        tok, st = engine.sample_logits(z, st, params, recent=seq)
        assert tok == t
        seq.append(tok)
        z = m.forward_one(tok, c)
    assert st == state
    m.close()


# -------------------------------------------------------------------------------- trace replay
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay(tmp_path, dtype):
    config, rows, rank = configs()["mixed"]
    path, ten = build(tmp_path / "m", config, 24, rows, rank)
    a, b = ids(18, 50, config["vocab"]), ids(19, 20, config["vocab"])
    steps = [{"entries": [{"id": "a", "tokens": a[:30].tolist(), "want": [0, 29]}]},
             {"entries": [{"id": "a", "tokens": a[30:49].tolist(), "want": []}]},
             {"entries": [{"id": "a", "tokens": a[49:].tolist(), "want": [0]}], "end": ["a"]},
             {"entries": [{"id": "b", "tokens": b.tolist(), "want": [3, 19]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.Popen([os.path.join(root, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out), "--max-tokens", "50"],
                         stdin=subprocess.PIPE, stdout=subprocess.PIPE, text=True)
    for i, s in enumerate(steps):
        p.stdin.write(json.dumps(dict({"end": []}, step=i, **s)) + "\n")
        p.stdin.flush()
        line = p.stdout.readline()
        while line and line.strip() != f"done {i}":
            line = p.stdout.readline()
        assert line, "the replay ended early"
    p.stdin.close()
    assert p.wait(timeout=60) == 0
    read = lambda i: np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, config["vocab"])
    za, zb = NO.forward(config, ten, a), NO.forward(config, ten, b)
    tol = TOL[registry.DTYPES[dtype]]
    assert error(read(0), za[[0, 29]]) < tol and error(read(2), za[[49]]) < tol and error(read(3), zb[[3, 19]]) < tol
    assert not (out / "1.f32").exists()
    bad = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out)],
                         stdin=subprocess.DEVNULL, capture_output=True)
    assert bad.returncode not in (0, 3)


def test_the_familys_own_library_is_enough(tmp_path):
    """A process that loads only the component the registry names serves the model."""
    from ferrum_cpu_b200 import build as B
    config, rows, rank = configs()["odd"]
    path, ten = build(tmp_path, config, 25, rows, rank)
    B.build(component="nurinex")
    code = ("import sys; sys.path.insert(0, sys.argv[1])\n"
            "from ferrum_cpu_b200 import _lib, build, registry\n"
            "_lib.use(build.component_lib('nurinex'))\n"
            "m = registry.load(sys.argv[2], ctx=32)\n"
            "print(int(m.forward_tokens([1, 2, 3])[-1].argmax()))\n")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-c", code, root, path], capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    m = CudaNurinex(path, ctx=32)
    assert int(r.stdout) == int(m.forward_tokens([1, 2, 3])[-1].argmax())
    m.close()
