"""Small synthetic Zogevik models shared by the tests: configurations, weights that make single mechanisms visible, and
comparison helpers. The oracle is oracle/zogevik_oracle.py."""
import numpy as np

from ferrum_cpu_b200 import model_dir as MD
from oracle import zogevik_oracle as ZO
from tests.nurinex_models import error, ids

LAT, ATT, MOE = MD.zogevik_latent, MD.zogevik_attention, MD.experts_config
CODE = 20          # entries of the residual that routers read in most tests (model_dir.zogevik_tensors)


def configs():
    """name -> config: other sizes, orders of layers, windows and sharing patterns."""
    return {
        # both mixers, shared caches under another window and scale, layers without a feed-forward
        "mixed": MD.zogevik_config(300, 96, [
            ATT(heads=6, kv_heads=2, dim=24, vdim=40, rot=8, window=33, base=5000.0, mlp=MOE(9, 3, 80, 3, 2)),
            LAT(heads=3, dim=24, rot=8, rank=40, vdim=20, window=17, mlp=None),
            ATT(heads=4, kv_heads=2, dim=24, vdim=40, rot=8, window=70, base=5000.0, scale=0.31, kv_from=0, mlp=MOE(5, 2, 48)),
            LAT(heads=5, dim=16, rot=20, rank=72, vdim=48, window=64, base=100.0, mlp=MOE(8, 1, 32, 4, 1)),
            ATT(heads=2, kv_heads=1, dim=32, vdim=16, rot=32, window=None, mlp=None),
            ATT(heads=6, kv_heads=2, dim=24, vdim=40, rot=8, window=9, base=5000.0, kv_from=0, mlp=MOE(4, 4, 64, 2, 2)),
        ], eps=1e-3),
        # sizes that are no multiples of anything
        "odd": MD.zogevik_config(131, 77, [
            LAT(heads=3, dim=19, rot=6, rank=37, vdim=13, window=21, scale=0.4, mlp=MOE(7, 3, 33, 7, 4)),
            ATT(heads=5, kv_heads=5, dim=18, vdim=11, rot=10, window=50, base=77.5, scale=0.33, mlp=MOE(10, 5, 50, 5, 3)),
        ], eps=1e-6),
        # one of everything
        "ones": MD.zogevik_config(90, 32, [
            LAT(heads=1, dim=8, rot=2, rank=16, vdim=8, window=2, mlp=MOE(1, 1, 16)),
            ATT(heads=1, kv_heads=1, dim=6, vdim=10, rot=2, window=1, mlp=MOE(3, 1, 8, 1, 1)),
            ATT(heads=1, kv_heads=1, dim=6, vdim=10, rot=2, window=5, kv_from=1, mlp=MOE(6, 6, 20, 2, 2)),
        ]),
        # more heads than a decode block holds, latents of several chunks, many experts
        "wide": MD.zogevik_config(260, 160, [
            LAT(heads=20, dim=80, rot=32, rank=328, vdim=72, window=90, mlp=MOE(40, 9, 136, 8, 5)),
            ATT(heads=36, kv_heads=2, dim=72, vdim=100, rot=48, window=130, mlp=MOE(65, 4, 72, 13, 6)),
        ]),
        # more experts than are ranked by counting
        "many": MD.zogevik_config(120, 48, [
            ATT(heads=2, kv_heads=2, dim=16, vdim=24, rot=4, window=31, mlp=MOE(150, 6, 24, 5, 3)),
            LAT(heads=2, dim=16, rot=4, rank=24, vdim=16, window=45, mlp=MOE(140, 30, 16)),
        ]),
        # query tiles too wide to stay in shared memory, value heads of four chunks, nothing masked but the future
        "huge": MD.zogevik_config(150, 64, [
            ATT(heads=2, kv_heads=1, dim=520, vdim=256, rot=130, window=None, mlp=MOE(3, 2, 520)),
            LAT(heads=2, dim=136, rot=72, rank=200, vdim=200, window=None, mlp=None),
        ]),
    }


def build(tmp_path, config, seed=0, code=CODE, edit=None):
    """Writes the folder; returns (path, f32 tensors as the oracle reads them). edit(tensors f32 dict) may change them."""
    bits = MD.zogevik_tensors(config, seed=seed, code=code)
    ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in bits.items()}
    if edit is not None:
        edit(ten)
        bits = {n: MD.to_bf16(a).reshape(np.shape(a)) for n, a in ten.items()}
        ten = {n: MD.from_bf16(b).reshape(b.shape) for n, b in bits.items()}
    return MD.write(str(tmp_path), config, bits), ten


def needle(ten, config, query_token, key_token, score=14.0):
    """Makes query_token attend to key_token in layer 0 wherever it stands within the window: each of the two owns one entry of
    the residual, and the unrotated query and key dimensions answer to those entries with a common sign pattern."""
    d, m = config["width"], config["layers"][0]["mixer"]
    a, b = d - 2, d - 1
    ten["embed"][:, [a, b]] = 0.0
    ten["embed.norm"][[a, b]] = 1.0
    for token, c in ((query_token, a), (key_token, b)):
        ten["embed"][token, CODE:] *= 0.05
        ten["embed"][token, c] = np.sqrt(d)
    x = d ** 0.5 * 0.7                      # about what that entry holds once the embedding is normed
    rng = np.random.default_rng(5)
    sign = lambda n: rng.choice([-1.0, 1.0], size=n).astype(np.float32)
    H, dim = m["heads"], m["dim"]
    if "kv_rank" in m:
        v, u, r = sign(dim), sign(m["kv_rank"]), m["kv_rank"]
        wq = ten["l0.mix.q"].reshape(H, dim + m["rot_dim"], d)
        wq[:, :, a] = 0.0
        wq[:, :dim, a] = v * score / (x * dim * m["scale"])
        ten["l0.mix.dkv"][:, b] = 0.0
        ten["l0.mix.dkv"][:r, b] = u
        ten["l0.mix.uk"].reshape(H, dim, r)[:] += v[:, None] * u / r
    else:
        free = dim - m["rot"]["dims"]
        v = sign(free)
        for name, heads, c in (("q", H, a), ("k", m["kv_heads"], b)):
            w = ten[f"l0.mix.{name}"].reshape(heads, dim, d)
            w[:, :, c] = 0.0
            w[:, m["rot"]["dims"]:, c] = v
            ten[f"l0.mix.{name}.norm"][:] = np.sqrt(score / (m["scale"] * dim))
    return ten


__all__ = ["ATT", "CODE", "LAT", "MD", "MOE", "ZO", "build", "configs", "error", "ids", "needle"]
