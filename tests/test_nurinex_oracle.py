"""The Nurinex oracle on values worked out by hand or by another route, and the host side of the family:
folder reader, configuration checks, registry. No GPU."""
import json
import math
import os
import struct

import numpy as np
import pytest

from ferrum_cpu_b200 import FerrumCudaError, _lib, decoder, registry
from tests.nurinex_models import MD, NO, L, build, configs, ids


def test_buckets_by_counting_and_at_exact_powers():
    # 8 rows, far 64: rows 4..7 start where (n / 4)^4 reaches 16^k, that is at 4, 8, 16 and 32
    want = [0, 1, 2, 3] + [4] * 4 + [5] * 8 + [6] * 16 + [7] * 40
    assert [NO.distance_bucket(n, 8, 64) for n in range(len(want))] == want
    for rows, far in ((2, 5), (10, 90), (16, 240), (32, 129)):
        b = [NO.distance_bucket(n, rows, far) for n in range(2 * far)]
        assert b == sorted(b) and b[-1] == rows - 1 and b[far] == rows - 1
        half = rows // 2
        for n in range(half, far):                       # the floating-point formula, away from whole quotients
            f = math.log(n / half) / math.log(far / half) * (rows - half)
            if abs(f - round(f)) > 1e-6:
                assert b[n] == min(rows - 1, half + math.floor(f))


def test_softmax_sink_counts_once_and_has_no_value():
    w = NO.softmax_with_sink(np.array([0.0, math.log(3.0)]), math.log(4.0))
    assert np.allclose(w, [1 / 8, 3 / 8])


def test_query_temperature_steps():
    assert NO.query_temperature(0, 0.5, 4) == 1.0
    assert NO.query_temperature(2, 0.5, 4) == 1.0
    assert math.isclose(NO.query_temperature(3, 0.5, 4), 1 + 0.5 * math.log(2))
    assert math.isclose(NO.query_temperature(11, 0.5, 4), 1 + 0.5 * math.log(4))


def test_wkv_equals_its_closed_form():
    rng = np.random.default_rng(0)
    T, D = 9, 5
    r, k, v = rng.standard_normal((3, T, D))
    d, u = rng.uniform(0.1, 1.0, (T, D)), rng.standard_normal(D)
    o, S = NO.wkv(r, k, v, d, u)
    for t in range(T):
        want = (r[t] * u * k[t]).sum() * v[t]
        for s in range(t):
            want = want + (r[t] * np.prod(d[s + 1:t], axis=0) * k[s]).sum() * v[s]
        assert np.allclose(o[t], want)
    o2, S2 = NO.wkv(r[4:], k[4:], v[4:], d[4:], u, NO.wkv(r[:4], k[:4], v[:4], d[:4], u)[1])
    assert np.allclose(o2, o[4:]) and np.allclose(S2, S)


def test_xielu_and_token_shift():
    p, q = 0.3, -0.7
    sp, sq = math.log(1 + math.exp(p)), math.log(1 + math.exp(q))
    z = np.array([2.0, 0.0, -1.5])
    want = [sp * 4 + 1, 0.0, (0.5 + sq) * (math.exp(-1.5) - 1 + 1.5) - 0.75]
    assert np.allclose(NO.xielu(z, p, q), want)
    h = np.arange(6.0).reshape(3, 2)
    assert np.array_equal(NO.token_shift(h), [[0, 0], [0, 1], [2, 3]])


def test_oracle_is_causal():
    config, rows, rank = configs()["mixed"]
    ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in MD.nurinex_tensors(config, 3, rows, rank).items()}
    a = ids(1, 24, config["vocab"])
    b = a.copy()
    b[15:] = (b[15:] + 1) % config["vocab"]
    x, y = NO.forward(config, ten, a), NO.forward(config, ten, b)
    assert np.array_equal(x[:15], y[:15]) and not np.allclose(x[15], y[15])


# ---------------------------------------------------------------------------------- host side
@pytest.mark.parametrize("name", sorted(configs()))
def test_probe_reads_every_configuration(tmp_path, name):
    config, rows, rank = configs()[name]
    path, _ = build(tmp_path, config, bias_rows=rows, rank=rank)
    info = decoder.probe(path)
    assert (info.vocab, info.width, info.n_layers) == (config["vocab"], config["width"], len(config["layers"]))
    assert info.n_own_layers == sum("weights_of" not in e for e in config["layers"])
    assert registry.architecture(path) == "Nurinex" and "Nurinex" in registry.ARCHITECTURES


def _edit_config(path, change):
    file = os.path.join(path, "config.json")
    config = json.load(open(file))
    change(config)
    json.dump(config, open(file, "w"))


BAD = {
    "architecture": (lambda c: c.update(architecture="Other"), _lib.FC_E_FORMAT),
    "layer type": (lambda c: c["layers"][0].update(type="serial"), _lib.FC_E_FORMAT),
    "feed-forward kind": (lambda c: c["layers"][0]["mlp"].update(kind="gated"), _lib.FC_E_FORMAT),
    "missing size": (lambda c: c["layers"][0]["mixer"]["left"].pop("heads"), _lib.FC_E_FORMAT),
    "heads that do not divide": (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=2), _lib.FC_E_DIM),
    "wrong width": (lambda c: c.update(width=80), _lib.FC_E_DIM),
    "wrong feed-forward": (lambda c: c["layers"][0]["mlp"].update(ff=99), _lib.FC_E_DIM),
    "circle": (lambda c: (c["layers"][0].update(weights_of=2), c["layers"][2].update(weights_of=0)), _lib.FC_E_FORMAT),
    "no such layer": (lambda c: c["layers"][0].update(weights_of=9), _lib.FC_E_FORMAT),
    "borrowed sizes": (lambda c: c["layers"][2].update(weights_of=1), _lib.FC_E_DIM),
    "bias range": (lambda c: [e["mixer"]["left"].update(bias_max=3) for e in c["layers"]], _lib.FC_E_DIM),
    "temperature step": (lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=0), _lib.FC_E_DIM),
}


@pytest.mark.parametrize("what", sorted(BAD))
def test_bad_configurations_are_refused_before_a_gpu_is_touched(tmp_path, what):
    config, rows, rank = configs()["mixed"]
    path, _ = build(tmp_path, config, bias_rows=rows, rank=rank)
    change, code = BAD[what]
    _edit_config(path, change)
    with pytest.raises(FerrumCudaError) as e:
        decoder.probe(path)
    assert e.value.code == code, str(e.value)


def test_bad_tensor_files_are_refused(tmp_path):
    config, rows, rank = configs()["mixed"]
    path, _ = build(tmp_path, config, bias_rows=rows, rank=rank)
    file = os.path.join(path, "model.safetensors")
    whole = open(file, "rb").read()
    n = struct.unpack("<Q", whole[:8])[0]
    head = json.loads(whole[8:8 + n])

    def refused(data):
        open(file, "wb").write(data)
        with pytest.raises(FerrumCudaError) as e:
            decoder.probe(path)
        return e.value.code

    def with_head(h):
        t = json.dumps(h).encode()
        return struct.pack("<Q", len(t)) + t + whole[8 + n:]

    assert refused(whole[:5]) == _lib.FC_E_FORMAT                       # no length
    assert refused(whole[:8 + n // 2]) == _lib.FC_E_FORMAT              # directory cut off
    assert refused(whole[:-64]) == _lib.FC_E_FORMAT                     # data cut off
    assert refused(struct.pack("<Q", 1 << 60) + whole[8:]) == _lib.FC_E_FORMAT
    h = dict(head)
    del h["final.norm"]
    assert refused(with_head(h)) == _lib.FC_E_FORMAT
    h = json.loads(json.dumps(head))
    h["head"]["shape"] = h["head"]["shape"][::-1]
    assert refused(with_head(h)) == _lib.FC_E_DIM
    h = json.loads(json.dumps(head))
    h["head"]["dtype"] = "F16"
    assert refused(with_head(h)) == _lib.FC_E_FORMAT
    h = json.loads(json.dumps(head))
    h["__metadata__"] = {"format": "pt", "note": "escapes \" \\ é \n"}
    open(file, "wb").write(with_head(h))
    decoder.probe(path)                                                  # metadata is skipped


def test_load_needs_a_gpu_and_a_mode_it_has(tmp_path):
    config, rows, rank = configs()["mixed"]
    path, _ = build(tmp_path, config, bias_rows=rows, rank=rank)
    with pytest.raises(FerrumCudaError) as e:
        decoder.CudaNurinex(path, math_mode=_lib.FC_MATH_BF16X3)
    assert e.value.code == _lib.FC_E_ARG
    if _lib.lib().fc_device_count() == 0:
        with pytest.raises(FerrumCudaError) as e:
            registry.load(path)
        assert e.value.code == _lib.FC_E_CUDA


def test_registry_knows_the_other_families(tmp_path):
    from ferrum_cpu_b200 import gguf_file, synth
    sm = synth.llama_named("llama-tiny")
    assert registry.architecture(gguf_file.write_llama_gguf(str(tmp_path / "m.gguf"), sm)) == "llama"
    with pytest.raises(FerrumCudaError):
        registry._gguf_mode(_lib.FC_MATH_BF16)


def test_component_sources_are_part_of_the_library():
    from ferrum_cpu_b200 import build as B
    for sources in B.COMPONENTS.values():
        assert set(sources) <= set(B.SOURCES) and len(set(sources)) == len(sources)
    assert {c for _, c in registry.ARCHITECTURES.values() if c} <= set(B.COMPONENTS)


def test_layer_template_matches_its_arguments():
    e = L(ff=0, weights_of=1)
    assert e["mlp"] is None and e["weights_of"] == 1
