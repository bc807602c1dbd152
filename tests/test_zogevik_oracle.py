"""The Zogevik oracle on values worked out by hand or by another route, and the host side of the family: configuration
checks, registry. No GPU."""
import copy
import json
import math
import os

import numpy as np
import pytest

from ferrum_cpu_b200 import FerrumCudaError, _lib, decoder, registry
from tests.zogevik_models import ATT, LAT, MD, MOE, ZO, build, configs, ids, needle


def test_rotations_turn_pairs_and_keep_distances():
    ang = ZO.angles([0, 3], 4, 100.0)
    assert np.allclose(ang, [[0, 0], [3.0, 0.3]])
    x = np.array([1.0, 0.0, 0.0, 2.0, 7.0])
    c, s = np.cos, np.sin
    assert np.allclose(ZO.rotate_neighbours(x[:4], ang[1]), [c(3), s(3), -2 * s(.3), 2 * c(.3)])
    assert np.allclose(ZO.rotate_halves(x, ang[1]), [c(3), -2 * s(.3), s(3), 2 * c(.3), 7])
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 12))
    for turn, dims in ((ZO.rotate_neighbours, 12), (ZO.rotate_halves, 8)):
        a = ZO.angles(range(40), dims, 50.0)
        dots = [turn(q, a[p + 5]) @ turn(k, a[p]) for p in range(30)]
        assert np.allclose(dots, dots[0]) and not np.isclose(dots[0], q @ k)


def test_windows_end_with_the_token():
    assert ZO.visible(5, 1).tolist() == [5]
    assert ZO.visible(5, 3).tolist() == [3, 4, 5]
    assert ZO.visible(2, 3).tolist() == [0, 1, 2] and ZO.visible(1, 3).tolist() == [0, 1]
    assert ZO.visible(3, None).tolist() == [0, 1, 2, 3]


def test_softmax_with_one_added():
    assert np.allclose(ZO.softmax_plus_one(np.log([2.0, 5.0])), [2 / 8, 5 / 8])
    assert np.allclose(ZO.softmax_plus_one(np.array([-800.0])), 0.0)
    assert np.allclose(ZO.softmax_plus_one(np.array([800.0, 800.0])), 0.5)
    assert np.allclose(ZO.softmax(np.log([2.0, 6.0])), [0.25, 0.75])


def test_routing_by_groups():
    z = np.log(np.array([5.0, 1.0, 4.0, 4.5, 0.5, 3.0]) / 18)
    r = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    chosen, w = ZO.route(z, r)                          # the first group holds the best one
    assert chosen == [0, 1] and np.allclose(w, [5 / 18, 1 / 18])
    chosen, w = ZO.route(z, dict(r, groups={"count": 3, "keep": 2}))
    assert chosen == [0, 3] and np.allclose(w, [5 / 18, 4.5 / 18])
    assert ZO.route(z, {"experts": 6, "top": 3})[0] == [0, 3, 2]
    chosen, w = ZO.route(z, {"experts": 6, "top": 6, "groups": {"count": 2, "keep": 2}})
    assert chosen == [0, 3, 2, 5, 1, 4] and np.isclose(w.sum(), 1.0)


def test_gelu_is_the_exact_form():
    z = np.array([-3.0, -0.5, 0.0, 1.0, 4.0])
    phi = np.array([0.0013498980316, 0.3085375387260, 0.5, 0.8413447460685, 0.9999683287582])
    assert np.allclose(ZO.gelu_erf(z), z * phi, atol=1e-10)


def test_latent_attention_equals_its_absorbed_form():
    """Queries carried into the latent space score the latents themselves, and values can be taken after the sum."""
    rng = np.random.default_rng(1)
    T, H, dim, rot, rank, vdim, d = 9, 2, 6, 4, 5, 3, 7
    w = {"q": rng.standard_normal((H * (dim + rot), d)), "dkv": rng.standard_normal((rank + rot, d)), "dkv.norm": rng.standard_normal(rank),
         "uk": rng.standard_normal((H * dim, rank)), "uv": rng.standard_normal((H * vdim, rank)), "o": rng.standard_normal((d, H * vdim))}
    cfg = {"heads": H, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "rot": {"base": 30.0, "dims": rot}, "scale": 0.4, "mask": {"size": 4}}
    h = rng.standard_normal((T, d))
    down = h @ w["dkv"].T
    c = down[:, :rank] / np.sqrt((down[:, :rank] ** 2).mean(1, keepdims=True) + 1e-5) * w["dkv.norm"]
    want = np.zeros((T, H, vdim))
    q = (h @ w["q"].T).reshape(T, H, dim + rot)
    for i in range(T):
        for n in range(H):
            qa = w["uk"].reshape(H, dim, rank)[n].T @ q[i, n, :dim]
            s = []
            for j in range(max(0, i - 3), i + 1):
                t = sum(((q[i, n, dim + 2 * a] + 1j * q[i, n, dim + 2 * a + 1]) * (down[j, rank + 2 * a] - 1j * down[j, rank + 2 * a + 1])
                         * np.exp(1j * (i - j) * 30.0 ** (-2 * a / rot))).real for a in range(rot // 2))
                s.append((qa @ c[j] + t) * 0.4)
            p = np.exp(s) / np.exp(s).sum()
            want[i, n] = w["uv"].reshape(H, vdim, rank)[n] @ (p @ c[max(0, i - 3):i + 1])
    assert np.allclose(ZO.latent_attention(h, w, cfg, 1e-5), want.reshape(T, -1) @ w["o"].T)


def test_oracle_is_causal_and_forgets_behind_its_windows():
    config = MD.zogevik_config(80, 32, [ATT(window=4, mlp=MOE(4, 2, 16)), LAT(window=3, mlp=None)])
    ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in MD.zogevik_tensors(config, 3).items()}
    a = ids(1, 24, 80)
    b = a.copy()
    b[10] = (b[10] + 1) % 80
    x, y = ZO.forward(config, ten, a), ZO.forward(config, ten, b)
    same = [bool(np.array_equal(u, v)) for u, v in zip(x, y)]
    assert same == [not 10 <= i <= 10 + 3 + 2 for i in range(24)]        # three tokens through one layer, two through the next


def test_needles_stand_out_in_the_oracle():
    for layer in (ATT(heads=4, kv_heads=2, dim=32, rot=8, window=12), LAT(heads=3, window=12)):
        config = MD.zogevik_config(60, 64, [layer])
        ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in MD.zogevik_tensors(config, 4, 20).items()}
        needle(ten, config, 7, 11)
        a = ids(2, 30, 60)
        a[(a == 7) | (a == 11)] = 5
        a[4] = 11
        for p, sees in ((15, True), (16, False)):
            x = a.copy()
            x[p] = 7
            y = x.copy()
            y[4] = 5
            diff = np.abs(ZO.forward(config, ten, x)[p] - ZO.forward(config, ten, y)[p]).max()
            assert diff > 0.3 if sees else diff == 0.0


# ---------------------------------------------------------------------------------- host side
@pytest.mark.parametrize("name", sorted(configs()))
def test_probe_reads_every_configuration(tmp_path, name):
    config = configs()[name]
    path, _ = build(tmp_path, config)
    info = decoder.probe(path)
    assert (info.vocab, info.width, info.n_layers) == (config["vocab"], config["width"], len(config["layers"]))
    assert info.n_own_layers == sum("kv_from" not in e["mixer"] for e in config["layers"])
    assert registry.architecture(path) == "Zogevik" and "Zogevik" in registry.ARCHITECTURES


def test_optional_entries_may_be_left_out(tmp_path):
    config = copy.deepcopy(configs()["mixed"])
    for e in config["layers"]:
        if e["mlp"] is None:
            del e["mlp"]
        elif e["mlp"]["router"]["groups"]["count"] == 1:
            del e["mlp"]["router"]["groups"]
        if e["mixer"]["mask"] is None:
            del e["mixer"]["mask"]
    assert decoder.probe(build(tmp_path, config)[0]).n_layers == 6


BAD = {
    "architecture": (lambda c: c.update(architecture="Other"), _lib.FC_E_FORMAT),
    "layer type": (lambda c: c["layers"][0].update(type="parallel"), _lib.FC_E_FORMAT),
    "feed-forward kind": (lambda c: c["layers"][0]["mlp"].update(kind="dense"), _lib.FC_E_FORMAT),
    "missing size": (lambda c: c["layers"][1]["mixer"].pop("kv_rank"), _lib.FC_E_FORMAT),
    "missing rotation": (lambda c: c["layers"][0]["mixer"].pop("rot"), _lib.FC_E_FORMAT),
    "missing router": (lambda c: c["layers"][0]["mlp"].pop("router"), _lib.FC_E_FORMAT),
    "empty window": (lambda c: c["layers"][0]["mixer"]["mask"].update(size=0), _lib.FC_E_FORMAT),
    "heads that do not divide": (lambda c: c["layers"][0]["mixer"].update(kv_heads=4), _lib.FC_E_DIM),
    "odd rotation": (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), _lib.FC_E_DIM),
    "more rotated than there is": (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=26), _lib.FC_E_DIM),
    "two rotated sizes": (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), _lib.FC_E_DIM),
    "wrong width": (lambda c: c.update(width=80), _lib.FC_E_DIM),
    "keys of a later layer": (lambda c: c["layers"][2]["mixer"].update(kv_from=3), _lib.FC_E_FORMAT),
    "keys of a latent layer": (lambda c: c["layers"][2]["mixer"].update(kv_from=1), _lib.FC_E_FORMAT),
    "keys of a layer that has none": (lambda c: c["layers"][5]["mixer"].update(kv_from=2), _lib.FC_E_FORMAT),
    "keys of another size": (lambda c: c["layers"][5]["mixer"].update(kv_from=4), _lib.FC_E_DIM),
    "keys of another rotation": (lambda c: c["layers"][2]["mixer"]["rot"].update(base=1.5), _lib.FC_E_DIM),
    "groups that do not divide": (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=2), _lib.FC_E_DIM),
    "too few to choose from": (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), _lib.FC_E_DIM),
    "more experts than there are": (lambda c: c["layers"][2]["mlp"]["router"].update(experts=6), _lib.FC_E_DIM),
}


@pytest.mark.parametrize("what", sorted(BAD))
def test_bad_configurations_are_refused_before_a_gpu_is_touched(tmp_path, what):
    path, _ = build(tmp_path, configs()["mixed"])
    change, code = BAD[what]
    file = os.path.join(path, "config.json")
    config = json.load(open(file))
    change(config)
    json.dump(config, open(file, "w"))
    with pytest.raises(FerrumCudaError) as e:
        decoder.probe(path)
    # a count the file's tensors contradict is found there
    assert e.value.code == code or (what == "more experts than there are" and e.value.code == _lib.FC_E_FORMAT), str(e.value)


def test_a_class_takes_folders_of_its_design_only(tmp_path):
    path, _ = build(tmp_path, configs()["ones"])
    with pytest.raises(FerrumCudaError) as e:
        decoder.CudaNurinex(path)
    assert e.value.code == _lib.FC_E_FORMAT
    with pytest.raises(FerrumCudaError) as e:
        decoder.CudaZogevik(path, math_mode=_lib.FC_MATH_BF16X3)
    assert e.value.code == _lib.FC_E_ARG
    assert math.isclose(LAT(dim=12, rot=4)["mixer"]["scale"], 0.25)
