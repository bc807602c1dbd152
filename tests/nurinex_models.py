"""Small synthetic Nurinex models shared by the tests: configurations, weights that make single mechanisms
visible, and comparison helpers. The oracle is oracle/nurinex_oracle.py."""
import numpy as np

from ferrum_cpu_b200 import model_dir as MD
from oracle import nurinex_oracle as NO

L = MD.nurinex_layer


def configs():
    """name -> (config, bias_rows, rank): other sizes, orders and sharing patterns."""
    return {
        # a bit of everything: sharing (also of a later layer's tensors), no feed-forward in one layer
        "mixed": (MD.nurinex_config(300, 96, [
            L(heads=4, kv_heads=2, dim=24, vdim=40, bias_max=90, every=13, r_heads=3, r_dim=32, ff=160),
            L(heads=3, kv_heads=1, dim=32, vdim=16, bias_max=37, coef=0.7, every=50, r_heads=2, r_dim=48, ff=0),
            L(heads=4, kv_heads=2, dim=24, vdim=40, bias_max=90, every=13, r_heads=3, r_dim=32, ff=160, weights_of=0),
            L(heads=3, kv_heads=1, dim=32, vdim=16, bias_max=37, coef=0.7, every=50, r_heads=2, r_dim=48, ff=0, weights_of=1),
        ], emb_scale=7.5), [10, 16, 0, 0], [5, 12, 0, 0]),
        # sizes that are no multiples of anything, one head, value width apart from key width
        "odd": (MD.nurinex_config(131, 76, [
            L(heads=5, kv_heads=5, dim=20, vdim=12, bias_max=33, every=7, r_heads=5, r_dim=20, ff=100, scale=0.31),
            L(heads=1, kv_heads=1, dim=6, vdim=10, bias_max=5, every=1, coef=0.2, r_heads=1, r_dim=7, ff=33),
        ], eps=1e-3, emb_scale=1.0), [2, 4], [1, 3]),
        # wide key rows: six k-chunks of the tensor-core attention, value heads of two chunks, groups of eight
        "wide": (MD.nurinex_config(520, 160, [
            L(heads=24, kv_heads=3, dim=128, vdim=72, bias_max=300, every=100, r_heads=2, r_dim=80, ff=256),
        ]), 32, 20),
        # a first layer that borrows a later one's tensors; many key/value heads; big recurrence heads
        "borrow": (MD.nurinex_config(200, 128, [
            L(heads=8, kv_heads=8, dim=16, vdim=32, bias_max=64, every=20, r_heads=1, r_dim=136, ff=64, weights_of=1),
            L(heads=8, kv_heads=8, dim=16, vdim=32, bias_max=64, every=20, r_heads=1, r_dim=136, ff=64),
        ], emb_scale=3.0), [0, 8], [0, 40]),
        # query tiles too wide to stay in shared memory, value heads of four chunks
        "huge": (MD.nurinex_config(150, 64, [
            L(heads=10, kv_heads=10, dim=120, vdim=200, bias_max=50, every=9, r_heads=1, r_dim=32, ff=64),
        ]), 6, 4),
    }


def build(tmp_path, config, seed=0, bias_rows=12, rank=8, edit=None):
    """Writes the folder; returns (path, f32 tensors as the oracle reads them). edit(tensors f32 dict) may change them."""
    bits = MD.nurinex_tensors(config, seed=seed, bias_rows=bias_rows, rank=rank)
    ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in bits.items()}
    if edit is not None:
        edit(ten)
        bits = {n: MD.to_bf16(a).reshape(np.shape(a)) for n, a in ten.items()}
        ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in bits.items()}
    return MD.write(str(tmp_path), config, bits), ten


def error(got, want):
    """Largest root-mean-square difference of a row of logits (means taken off) over the rows' typical size."""
    d = np.asarray(got, dtype=np.float64) - want
    d = d - d.mean(axis=-1, keepdims=True)
    scale = np.sqrt(np.mean((want - want.mean(axis=-1, keepdims=True)) ** 2))
    return float(np.sqrt((d ** 2).mean(axis=-1)).max() / scale)


def ids(seed, n, vocab):
    return np.random.default_rng(seed).integers(0, vocab, n).astype(np.int32)


def needle(ten, config, query_token, key_token, layer=0, strength=6.0):
    """Makes query_token attend to key_token wherever it stands: each token owns one direction of the normed stream, and
    the first query head of every group and every key head get those directions with a common sign pattern, so that this
    one score stands out by roughly strength^2. Talk, bias and sink stay as they are."""
    d = config["width"]
    l = config["layers"][layer]["mixer"]["left"]
    a, b = d // 2, d // 2 + 1
    size = 4.0 / max(config["embedding"]["scale"], 1e-6)
    ten["embed"][:, [a, b]] = 0.0
    for token, c in ((query_token, a), (key_token, b)):
        ten["embed"][token] *= 0.3
        ten["embed"][token, c] = size
    v = np.random.default_rng(99).choice([-1.0, 1.0], size=l["dim"]).astype(np.float32)
    per = l["heads"] // l["kv_heads"]
    wq = ten[f"l{layer}.mix.left.q"].reshape(l["heads"], l["dim"], d)
    wk = ten[f"l{layer}.mix.left.k"].reshape(l["kv_heads"], l["dim"], d)
    gain = strength / np.sqrt(d) / l["dim"] ** 0.25
    wq[::per, :, a] = v * gain
    wk[:, :, b] = v * gain
    return ten


__all__ = ["MD", "NO", "L", "configs", "build", "error", "ids", "needle"]
