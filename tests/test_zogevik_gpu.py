"""Zogevik on the GPU against the plain numpy oracle, in f32 (tight) and in bf16 (the precision it is served in): each
mechanism with its absence ruled out, prompts, decoding, portions, reused caches, keys at every window's edge, scoring and
generation through the serving front."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from ferrum_cpu_b200 import FerrumCudaError, _lib, engine, registry
from ferrum_cpu_b200.backend import CudaBackend, GenRequest
from ferrum_cpu_b200.decoder import CudaZogevik
from tests.zogevik_models import ATT, LAT, MD, MOE, ZO, build, configs, error, ids, needle

pytestmark = pytest.mark.gpu
F32, BF16 = _lib.FC_MATH_FP32, _lib.FC_MATH_BF16
TOL = {F32: 2e-5, BF16: 2.5e-2}
MODES = pytest.mark.parametrize("mode", [F32, BF16], ids=["f32", "bf16"])
MIXERS = pytest.mark.parametrize("kind", ["attention", "latent"])


def feed_in(model, cache, toks, cuts):
    """Logits of every token, fed in portions that end at `cuts`."""
    out, at = np.empty((len(toks), model.info.vocab), dtype=np.float32), 0
    for e in list(cuts) + [len(toks)]:
        if e > at:
            out[at:e] = model.feed(toks[at:e], cache, range(e - at))
            at = e
    return out


def check(path, config, ten, mode, toks, cuts=(), want=None, ctx=None):
    want = ZO.forward(config, ten, toks) if want is None else want
    m = CudaZogevik(path, math_mode=mode, ctx=ctx or len(toks))
    got = feed_in(m, m.new_cache(), toks, cuts)
    m.close()
    assert error(got, want) < TOL[mode], error(got, want)
    return got, want


# ------------------------------------------------------------------------------- whole models
@MODES
@pytest.mark.parametrize("name", sorted(configs()))
def test_prompt_decode_and_portions_match_the_oracle(tmp_path, name, mode):
    config = configs()[name]
    path, ten = build(tmp_path, config, 5)
    toks = ids(2, 150, config["vocab"])
    want = ZO.forward(config, ten, toks)
    m = CudaZogevik(path, math_mode=mode, ctx=160)
    c = m.new_cache()
    for cuts in ([], range(1, 150), [2, 4, 7, 12, 29, 31, 64, 66, 67, 128], [100] + list(range(101, 150)), range(2, 150, 2)):
        c.clear()
        got = feed_in(m, c, toks, cuts)
        assert c.pos() == 150
        assert error(got, want) < TOL[mode], (list(cuts)[:4], error(got, want))
    m.close()


def test_routing_that_hangs_on_the_whole_residual(tmp_path):
    """Routers that read every entry, in f32: what came before decides which experts a token uses."""
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 6, code=0)
    toks = ids(3, 120, config["vocab"])
    for cuts in ([], range(40, 120)):
        check(path, config, ten, F32, toks, cuts)


@MODES
def test_residual_stream_after_every_layer(tmp_path, mode):
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 6)
    toks = ids(3, 40, config["vocab"])
    lay = []
    ZO.forward(config, ten, toks, lay)
    m = CudaZogevik(path, math_mode=mode, ctx=64)
    c = m.new_cache()
    got = np.concatenate([m.feed_layers(toks[:23], c), m.feed_layers(toks[23:], c)], axis=1)
    for i, w in enumerate(lay):
        assert np.abs(got[i] - w).max() < (2e-6 if mode == F32 else 2e-2) * np.abs(w).max(), i
    m.close()


@MODES
def test_portions_do_not_change_the_logits(tmp_path, mode):
    """Beyond rounding the cut does not matter: not in portions, nor token by token."""
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 7)
    toks = ids(4, 300, config["vocab"])
    m = CudaZogevik(path, math_mode=mode, ctx=300)
    c = m.new_cache()
    whole = feed_in(m, c, toks, [])
    for cuts in ([128], [63, 65, 191], [2, 298], [7 * k for k in range(1, 42)]):
        c.clear()
        assert error(feed_in(m, c, toks, cuts), whole) < TOL[mode] / 4, cuts
    c.clear()
    assert error(feed_in(m, c, toks, range(250, 300)), whole) < TOL[mode]
    m.close()


# --------------------------------------------------------------------- one mechanism at a time
def one_layer(kind, window=25, mlp=None, eps=1e-2, **kw):
    layer = (ATT(heads=6, kv_heads=2, dim=32, vdim=24, rot=12, window=window, base=900.0, scale=0.35, mlp=mlp, **kw) if kind == "attention"
             else LAT(heads=6, dim=32, rot=12, rank=48, vdim=24, window=window, base=900.0, scale=0.35, mlp=mlp, **kw))
    return MD.zogevik_config(180, 72, [layer], eps=eps)


rotate_halves, rotate_neighbours, visible, route, rms = ZO.rotate_halves, ZO.rotate_neighbours, ZO.visible, ZO.route, ZO.rms_norm
MECHANISMS = {
    # name: (mixer, feed-forward, the oracle without the mechanism as (function, replacement))
    "sink": ("attention", None, ("softmax_plus_one", ZO.softmax)),
    "no sink in latent attention": ("latent", None, ("softmax", ZO.softmax_plus_one)),
    "window one too long": ("attention", None, ("visible", lambda i, w: visible(i, w + 1))),
    "window one too short": ("latent", None, ("visible", lambda i, w: visible(i, w - 1))),
    "rotation of halves": ("attention", None, ("rotate_halves", lambda x, a: np.concatenate([rotate_neighbours(x[..., :12], a), x[..., 12:]], -1))),
    "rotation of neighbours": ("latent", None, ("rotate_neighbours", rotate_halves)),
    "positions count from 0": ("attention", None, ("angles", lambda p, d, b, f=ZO.angles: f(p, d, b) * 1.02)),
    "norm of queries and keys over the projection": ("attention", None, ("keys_and_values", lambda h, w, cfg, eps: (
        rotate_halves(rms(ZO.linear(w["k"], h).reshape(len(h), 2, 32), w["k.norm"].reshape(2, 32), eps), ZO.angles(range(len(h)), 12, 900.0)[:, None]),
        ZO.linear(w["v"], h).reshape(len(h), 2, 24)))),
    "groups of experts": ("latent", MOE(8, 2, 40, 4, 1), ("route", lambda z, r: route(z, dict(r, groups=None)))),
    "weights not renormalised": ("attention", MOE(8, 2, 40, 4, 2), ("route", lambda z, r: (route(z, r)[0], route(z, r)[1] * [0.5, 2.0]))),
    "exact gelu": ("attention", MOE(8, 2, 40, 4, 2), ("gelu_erf", lambda z: np.maximum(z, 0))),
}


@MODES
@pytest.mark.parametrize("what", sorted(MECHANISMS))
def test_each_mechanism_shows(tmp_path, monkeypatch, what, mode):
    kind, mlp, (fn, without) = MECHANISMS[what]
    config = one_layer(kind, mlp=mlp, window=6 if "window" in what else 25)

    def edit(ten):
        if mlp:                                            # the feed-forward outweighs the mixer
            ten["l0.norm1"] *= 0.2
            ten["l0.norm2"] *= 2.0
    path, ten = build(tmp_path, config, 8, edit=edit)
    toks = ids(5, 90, config["vocab"])
    for cuts in ([], range(30, 90)):
        got, _ = check(path, config, ten, mode, toks, cuts)
    monkeypatch.setattr(ZO, fn, without)
    assert error(got, ZO.forward(config, ten, toks)) > 2 * TOL[mode]       # an oracle without it is told apart


@MIXERS
def test_every_small_tensor_reaches_the_result(tmp_path, kind):
    """f32: matches the oracle, and an oracle with that tensor's entries turned round does not match."""
    config = one_layer(kind, mlp=MOE(5, 2, 40))
    toks = ids(6, 60, config["vocab"])
    path, ten = build(tmp_path, config, 9)
    got, _ = check(path, config, ten, F32, toks)
    for name in sorted(n for n in ten if n.endswith(("norm", "norm1", "norm2", "router")) or ".e3." in n):
        changed = dict(ten, **{name: np.ascontiguousarray(ten[name].ravel()[::-1].reshape(ten[name].shape))})
        assert error(got, ZO.forward(config, changed, toks)) > 50 * TOL[F32], name


@MIXERS
def test_constants_are_read_from_the_configuration(tmp_path, kind):
    toks = ids(7, 70, 180)
    base = one_layer(kind, mlp=MOE(12, 4, 40, 4, 2))

    def variant(eps=None, router=None, **mixer):
        c = copy.deepcopy(base)
        c["layers"][0]["mixer"].update(mixer)
        c["layers"][0]["mlp"]["router"].update(router or {})
        if eps:
            c["norm"]["eps"] = eps
        return c
    rot = base["layers"][0]["mixer"]["rot"]
    cases = [base, variant(scale=0.05), variant(mask={"size": 24}), variant(mask=None), variant(rot=dict(rot, base=30.0)), variant(eps=1e-6),
             variant(router={"top": 3}), variant(router={"groups": {"count": 3, "keep": 1}}), variant(router={"groups": {"count": 4, "keep": 4}})]
    if kind == "attention":
        cases.append(variant(rot=dict(rot, dims=32)))
    _, ten = build(tmp_path / "w", base, 10)
    results = []
    for i, c in enumerate(cases):
        p = MD.write(str(tmp_path / str(i)), c, {n: MD.to_bf16(a).reshape(a.shape) for n, a in ten.items()})
        results.append(check(p, c, ten, F32, toks, range(40, 70))[0])
    for i in range(1, len(cases)):
        assert error(results[i], results[0]) > 20 * TOL[F32], i


@MODES
def test_activation_on_both_sides_and_far_out(tmp_path, mode):
    config = one_layer("attention", mlp=MOE(4, 2, 64))

    def edit(ten):
        for e in range(4):
            ten[f"l0.mlp.e{e}.up"] *= 4                    # arguments from about -20 to 20
    path, ten = build(tmp_path, config, 11, edit=edit)
    check(path, config, ten, mode, ids(8, 50, config["vocab"]), range(25, 50))


@MODES
def test_every_expert_and_every_token_of_one_expert(tmp_path, mode):
    """A router that sends all tokens to the same experts (runs of hundreds of rows, experts without any), and one that spreads
    them; a run's rows cross the row tiles of the products."""
    config = one_layer("attention", mlp=MOE(30, 3, 48, 6, 3))
    for name, gain in (("same", 0.0), ("spread", 3.0)):
        def edit(ten):
            r = ten["l0.mlp.router"]
            r *= gain
            ten["embed"][:, 0] = 4.0                       # one entry all tokens share decides, or does nothing
            r[:, 0] = 0.0 if gain else np.linspace(-1.0, 1.0, 30)[np.random.default_rng(0).permutation(30)]
        path, ten = build(tmp_path / name, config, 12, edit=edit)
        toks = ids(9, 430, config["vocab"])
        used = {e for t in np.unique(toks) for e in ZO.route(ten["l0.mlp.router"] @ ZO.rms_norm(ten["embed"][t], ten["embed.norm"], 1e-2), config["layers"][0]["mlp"]["router"])[0]}
        assert (len(used) == 3) if name == "same" else (len(used) > 20)
        check(path, config, ten, mode, toks, [300, 302] + list(range(420, 430)))


# ------------------------------------------------------------------ far keys, edges, first tokens
@MODES
@MIXERS
@pytest.mark.parametrize("window", [2, 16, 63, 64, 65, 100, 128, 200, 300])
def test_keys_just_inside_and_just_outside_the_window(tmp_path, kind, window, mode):
    """One token attends to another one; in the window's last place it is found, one further on it is not. The asking token
    stands in a prompt, alone in a decode step, and at the start, middle and end of a portion."""
    base = one_layer(kind, window=window)
    asks, holds, first = 7, 11, 5
    path, ten = build(tmp_path, base, 13, edit=lambda t: needle(t, base, asks, holds))
    T = window + 140
    toks = ids(10, T, base["vocab"])
    toks[(toks == asks) | (toks == holds)] = 8
    m = CudaZogevik(path, math_mode=mode, ctx=T)
    for at in (first, first + 123):                        # the key at two places: tile borders fall differently
        for p, seen in ((at + window - 1, True), (at + window, False)):
            a = toks.copy()
            a[at] = holds
            a[p] = asks
            a = a[:p + 3]
            want = ZO.forward(base, ten, a)
            b = a.copy()
            b[at] = 9
            other = ZO.forward(base, ten, b)
            assert (error(want[p:p + 1], other[p:p + 1]) > 3 * TOL[mode]) == seen
            for cuts in ([], [p], [p, p + 1], [p - 1], [p // 2]):
                got = feed_in(m, m.new_cache(), a, cuts)
                assert error(got[p:p + 1], want[p:p + 1]) < TOL[mode], (p, cuts)
    m.close()


@MODES
@MIXERS
def test_a_far_key_is_found_at_every_distance(tmp_path, kind, mode):
    """Without a window: distances on tile and split edges, among hundreds of other keys."""
    base = one_layer(kind, window=None)
    asks, holds, T, first = 7, 11, 420, 5
    path, ten = build(tmp_path, base, 14, edit=lambda t: needle(t, base, asks, holds))
    toks = ids(10, T, base["vocab"])
    toks[(toks == asks) | (toks == holds)] = 8
    toks[first] = holds
    m = CudaZogevik(path, math_mode=mode, ctx=T)
    for p in sorted({first + n for n in (1, 3, 31, 32, 33, 58, 59, 60, 63, 64, 65, 127, 128, 129, 255, 256, 257, 400)}):
        a = toks.copy()
        a[p] = asks
        a = a[:p + 3]
        want = ZO.forward(base, ten, a)
        b = a.copy()
        b[first] = 9
        assert error(want[p:p + 1], ZO.forward(base, ten, b)[p:p + 1]) > 3 * TOL[mode], p      # the far key matters
        for cuts in ([], [p], [p, p + 1]):
            assert error(feed_in(m, m.new_cache(), a, cuts)[p:p + 1], want[p:p + 1]) < TOL[mode], (p, cuts)
    m.close()


@MODES
def test_shared_keys_under_a_window_of_their_own(tmp_path, mode):
    """The layer that borrows keys sees further back, or less far, than the layer that made them."""
    for own, borrowed in ((8, 90), (90, 8), (40, 40)):
        config = MD.zogevik_config(160, 64, [ATT(heads=4, kv_heads=2, rot=8, window=own),
                                             ATT(heads=8, kv_heads=2, rot=8, window=borrowed, scale=0.3, kv_from=0)])
        path, ten = build(tmp_path / f"{own}-{borrowed}", config, 15)
        toks = ids(11, 140, 160)
        for cuts in ([], [1, 3, 70] + list(range(100, 140))):
            check(path, config, ten, mode, toks, cuts)


@MODES
def test_first_tokens_and_single_token_sequences(tmp_path, mode):
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 16)
    m = CudaZogevik(path, math_mode=mode, ctx=8)
    c = m.new_cache()
    for n in (1, 2, 3, 5):
        toks = ids(20 + n, n, config["vocab"])
        want = ZO.forward(config, ten, toks)
        for cuts in ([], [1], range(1, n)):
            c.clear()
            assert error(feed_in(m, c, toks, cuts), want) < TOL[mode]
    m.close()


@MODES
def test_long_decoding(tmp_path, mode):
    """Past many windows and splits, token by token from a short prompt."""
    config = MD.zogevik_config(180, 72, [one_layer(k, window=w)["layers"][0] for k, w in (("attention", 70), ("latent", 200), ("attention", None), ("latent", None))])
    path, ten = build(tmp_path, config, 17)
    toks = ids(11, 500, config["vocab"])
    check(path, config, ten, mode, toks, range(3, 500), ctx=4500)


def test_positions_far_out(tmp_path):
    """f32: angles of positions in the tens of thousands keep their precision; logits behind a window depend on distances only,
    so a repeated sequence repeats its logits."""
    config = MD.zogevik_config(50, 32, [one_layer(k, window=20)["layers"][0] for k in ("attention", "latent")])
    path, ten = build(tmp_path, config, 18)
    unit = ids(12, 500, 50)
    toks = np.tile(unit, 70)
    m = CudaZogevik(path, math_mode=F32, ctx=35000)
    c = m.new_cache()
    m.feed(toks[:34900], c)
    got = feed_in(m, c, toks[34900:], [20, 30] + list(range(60, 70)))
    want = ZO.forward(config, ten, unit)[400:]
    assert error(got, want) < 5 * TOL[F32]
    m.close()


# ------------------------------------------------------------------------ caches, reuse, refusals
@MODES
def test_caches_are_independent_and_reusable(tmp_path, mode):
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 19)
    m = CudaZogevik(path, math_mode=mode, ctx=130)
    seqs = [ids(30 + i, n, config["vocab"]) for i, n in enumerate((130, 3, 57))]
    alone = []
    c = m.new_cache()
    for s in seqs:                                   # one cache for all, longest first: what it held must not show
        c.clear()
        alone.append(feed_in(m, c, s, []))
        assert error(alone[-1], ZO.forward(config, ten, s)) < TOL[mode]
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
    config = configs()["odd"]
    path, ten = build(tmp_path, config, 20)
    m = CudaZogevik(path, math_mode=F32, ctx=20)
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
    assert error(got, ZO.forward(config, ten, toks)[10:]) < TOL[F32]
    with pytest.raises(FerrumCudaError):
        m.feed([1], c)                                     # full
    m.close()


@MODES
def test_portions_longer_than_one_pass(tmp_path, mode):
    """More tokens than a forward pass takes are cut inside the call; nothing shows at the seam."""
    config = MD.zogevik_config(90, 32, [ATT(heads=2, kv_heads=1, dim=16, vdim=16, rot=8, window=70, mlp=MOE(4, 2, 32)), LAT(heads=2, window=150)])
    path, ten = build(tmp_path, config, 21)
    toks = ids(13, 2300, 90)
    m = CudaZogevik(path, math_mode=mode, ctx=2300)
    c = m.new_cache()
    places = [0, 2046, 2047, 2048, 2049, 2299]
    a = m.feed(toks, c, places)
    c.clear()
    m.feed(toks[:1000], c)
    b = m.feed(toks[1000:], c, [p - 1000 for p in places[1:]])
    assert error(b, a[1:]) < TOL[mode] / 4
    assert error(a, ZO.forward(config, ten, toks)[places]) < TOL[mode]
    m.close()


def test_waits_that_run_out_are_reported(tmp_path):
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 22)
    m = CudaZogevik(path, math_mode=BF16, ctx=64)
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
    assert error(feed_in(m, c, toks, []), ZO.forward(config, ten, toks)) < TOL[BF16]
    m.close()


# ------------------------------------------------------------------------- scoring and generation
@MODES
def test_scoring_matches_the_oracle(tmp_path, mode):
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 23)
    be = CudaBackend(registry.load(path, math_mode=mode, ctx=200))
    assert isinstance(be.model, CudaZogevik)
    toks = ids(15, 120, config["vocab"])
    z = ZO.forward(config, ten, toks)
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
    config = configs()["mixed"]
    path, ten = build(tmp_path, config, 24)
    be = CudaBackend(registry.load(path, math_mode=F32, ctx=128))
    prompt = ids(16, 19, config["vocab"]).tolist()
    seq, margins = list(prompt), []
    for _ in range(60):                              # past several windows
        z = ZO.forward(config, ten, seq)[-1]
        top = np.sort(z)
        margins.append(top[-1] - top[-2])
        seq.append(int(z.argmax()))
    assert min(margins) > 1e-4
    want = seq[19:]
    for n in (1, 60):
        assert be.generate(GenRequest(prompt, max_tokens=n, temperature=0.0))["tokens"] == want[:n]
    eos = want[12]
    stop = want.index(eos)
    assert be.generate(GenRequest(prompt, max_tokens=30, temperature=0.0, eos=eos))["tokens"] == want[:stop]
    one = be.generate(GenRequest(prompt[:1], max_tokens=5, temperature=0.0))["tokens"]      # a one-token prompt
    seq = prompt[:1]
    for _ in range(5):
        seq.append(int(ZO.forward(config, ten, seq)[-1].argmax()))
    assert one == seq[1:]
    long = be.generate(GenRequest(prompt, max_tokens=500, temperature=0.0))["tokens"]       # ends with the context
    assert len(long) == 128 - 19 and long[:60] == want
    req = GenRequest(prompt, max_tokens=20, temperature=0.9, top_k=20, seed=3)
    assert be.generate(req) == be.generate(req)
    assert be.generate(GenRequest(prompt, cancel=np.ones(1, np.int32))) is None
    be.model.close()


def test_sampling_with_penalty_equals_the_sampler_on_the_logits(tmp_path):
    config = configs()["odd"]
    path, ten = build(tmp_path, config, 25)
    m = CudaZogevik(path, math_mode=F32, ctx=64)
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
    config = configs()["mixed"]
    path, ten = build(tmp_path / "m", config, 26)
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
    za, zb = ZO.forward(config, ten, a), ZO.forward(config, ten, b)
    tol = TOL[registry.DTYPES[dtype]]
    assert error(read(0), za[[0, 29]]) < tol and error(read(2), za[[49]]) < tol and error(read(3), zb[[3, 19]]) < tol


def test_the_familys_own_library_is_enough(tmp_path):
    """A process that loads only the component the registry names serves the model."""
    from ferrum_cpu_b200 import build as B
    config = configs()["odd"]
    path, ten = build(tmp_path, config, 27)
    B.build(component="zogevik")
    code = ("import sys; sys.path.insert(0, sys.argv[1])\n"
            "from ferrum_cpu_b200 import _lib, build, registry\n"
            "_lib.use(build.component_lib('zogevik'))\n"
            "m = registry.load(sys.argv[2], ctx=32)\n"
            "print(int(m.forward_tokens([1, 2, 3])[-1].argmax()))\n")
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, "-c", code, root, path], capture_output=True, text=True)
    assert r.returncode == 0, r.stderr
    m = CudaZogevik(path, ctx=32)
    assert int(r.stdout) == int(m.forward_tokens([1, 2, 3])[-1].argmax())
    m.close()
