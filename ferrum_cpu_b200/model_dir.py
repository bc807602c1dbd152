"""Writer of model folders (config.json + model.safetensors) and synthetic models of the designs, for tests and
benchmarks. Reading is the library's (csrc/model_dir.cpp)."""
import json
import os
import struct

import numpy as np


def to_bf16(a):
    """f32 array -> uint16 bf16 bits, round to nearest even."""
    u = np.ascontiguousarray(a, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(bits):
    return (np.ascontiguousarray(bits, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)


def write(path, config, tensors):
    """tensors: name -> uint16 array of bf16 bits (shape kept)."""
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(config, f, indent=1)
    head, at = {}, 0
    for name, a in tensors.items():
        head[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + a.nbytes]}
        at += a.nbytes
    text = json.dumps(head).encode()
    with open(os.path.join(path, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(text)))
        f.write(text)
        for a in tensors.values():
            f.write(np.ascontiguousarray(a).tobytes())
    return path


def nurinex_layer(heads=4, kv_heads=2, dim=32, vdim=32, bias_max=100, scale=None, coef=0.3, every=16, r_heads=3, r_dim=32, ff=96,
                  weights_of=None):
    """One entry of `layers`. ff 0: no feed-forward."""
    entry = {
        "type": "parallel",
        "mixer": {
            "left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max,
                     "scale": dim ** -0.5 if scale is None else scale, "q_temp": {"coef": coef, "every": every}},
            "right": {"heads": r_heads, "dim": r_dim},
        },
        "mlp": {"kind": "dense", "ff": ff} if ff else None,
    }
    if weights_of is not None:
        entry["weights_of"] = weights_of
    return entry


def nurinex_config(vocab, width, layers, eps=1e-5, emb_scale=1.0):
    return {"architecture": "Nurinex", "vocab": vocab, "width": width, "embedding": {"scale": emb_scale}, "norm": {"eps": eps}, "layers": layers}


# name -> (vocab, width, layers, query heads, key/value heads, head dim, recurrence heads, recurrence dim, ff, decay rank):
# layers as those of real models, few of them. The first has the layer sizes of the 1B-class Llama shape in synth.py.
NURINEX_SHAPES = {
    "nurinex-small": (32000, 1024, 12, 16, 4, 64, 16, 64, 4096, 32),
    "nurinex-1b": (32000, 2048, 8, 32, 8, 64, 32, 64, 8192, 64),
    "nurinex-7b-layers": (32000, 4096, 3, 32, 8, 128, 64, 64, 11008, 64),
}


def nurinex_named(path, name, seed=0):
    """Writes a synthetic model of a named shape; returns its configuration."""
    V, d, n, H, G, hd, rH, rD, ff, rank = NURINEX_SHAPES[name]
    layer = nurinex_layer(heads=H, kv_heads=G, dim=hd, vdim=hd, bias_max=1024, every=512, r_heads=rH, r_dim=rD, ff=ff)
    config = nurinex_config(V, d, [layer] * n)
    write(path, config, nurinex_tensors(config, seed=seed, bias_rows=32, rank=rank))
    return config


def nurinex_tensors(config, seed=0, bias_rows=12, rank=8):
    """Random bf16 weights of the shapes a configuration asks for: name -> uint16 array. bias_rows and rank are numbers
    or one per layer."""
    rng = np.random.default_rng(seed)
    d, V = config["width"], config["vocab"]
    out = {}

    def put(name, shape, std, mean=0.0):
        out[name] = to_bf16(rng.standard_normal(shape, dtype=np.float32) * np.float32(std) + np.float32(mean))

    put("embed", (V, d), 1.0 / max(config["embedding"]["scale"], 1e-6))
    for i, layer in enumerate(config["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, l, r = f"l{i}.", layer["mixer"]["left"], layer["mixer"]["right"]
        rows = bias_rows[i] if isinstance(bias_rows, (list, tuple)) else bias_rows
        rk = rank[i] if isinstance(rank, (list, tuple)) else rank
        H, G, rd = l["heads"], l["kv_heads"], r["heads"] * r["dim"]
        put(p + "norm1", (d,), 0.2, 1.0)
        put(p + "mix.left.q", (H * l["dim"], d), d ** -0.5 * 1.5)
        put(p + "mix.left.k", (G * l["dim"], d), d ** -0.5 * 1.5)
        put(p + "mix.left.v", (G * l["vdim"], d), d ** -0.5)
        put(p + "mix.left.rel", (rows, H), 1.0)
        out[p + "mix.left.talk"] = to_bf16(np.eye(H, dtype=np.float32) + rng.standard_normal((H, H), dtype=np.float32) * np.float32(0.25))
        put(p + "mix.left.sink", (H,), 1.0, 1.0)
        put(p + "mix.left.o", (d, H * l["vdim"]), (H * l["vdim"]) ** -0.5)
        for s in "rkvgw":
            put(p + "mix.right.mu." + s, (d,), 0.25, 0.5)
        for s in "rkvg":
            put(p + "mix.right." + s, (rd, d), d ** -0.5)
        put(p + "mix.right.w1", (rk, d), d ** -0.5)
        put(p + "mix.right.w2", (rd, rk), rk ** -0.5)
        put(p + "mix.right.w0", (rd,), 1.5, -3.0)
        put(p + "mix.right.u", (r["heads"], r["dim"]), 0.5, 0.5)
        put(p + "mix.right.norm", (rd,), 0.2, 1.0)
        put(p + "mix.right.o", (d, rd), rd ** -0.5)
        put(p + "mix.left.out", (d,), 0.2, 1.0)
        put(p + "mix.right.out", (d,), 0.2, 1.0)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            put(p + "mlp.up", (ff, d), d ** -0.5)
            put(p + "mlp.down", (d, ff), ff ** -0.5)
            put(p + "mlp.act", (2,), 0.5, 0.3)
    put("final.norm", (d,), 0.2, 1.0)
    put("head", (V, d), d ** -0.5)
    return out


def experts_config(experts=8, top=2, ff=64, groups=1, keep=1):
    """The routed feed-forward of a Zogevik layer."""
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "groups": {"count": groups, "keep": keep}}}


def zogevik_latent(heads=4, dim=32, rot=16, rank=64, vdim=32, window=40, base=10000.0, scale=None, mlp=None):
    """One entry of `layers`: latent attention. window None: all earlier positions; mlp None: no feed-forward."""
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot, "kv_rank": rank, "vdim": vdim, "rot": {"base": base, "dims": rot},
             "scale": (dim + rot) ** -0.5 if scale is None else scale, "mask": None if window is None else {"size": window}}
    return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


def zogevik_attention(heads=4, kv_heads=2, dim=32, vdim=32, rot=16, window=40, base=10000.0, scale=None, kv_from=None, mlp=None):
    """One entry of `layers`: grouped-query attention; kv_from: the layer whose keys and values it uses."""
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": rot},
             "scale": dim ** -0.5 if scale is None else scale, "mask": None if window is None else {"size": window}}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    return {"type": "attention", "mixer": mixer, "mlp": mlp}


def zogevik_config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Zogevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


# name -> (vocab, width, layers, latent (heads, dim, rotated, rank, value dim), grouped-query (heads, kv heads, dim, rotated), window,
# (experts, chosen, ff of one, groups, kept)): layers as those of real models, few of them; every third is grouped-query, and
# every second of those uses the keys of the one before.
ZOGEVIK_SHAPES = {
    "zogevik-small": (32000, 1024, 12, (16, 64, 32, 256, 64), (16, 4, 64, 64), 1024, (32, 8, 512, 4, 2)),
    "zogevik-1b": (32000, 2048, 8, (16, 128, 64, 512, 128), (32, 8, 64, 64), 1024, (32, 8, 1024, 4, 2)),
    "zogevik-7b-layers": (32000, 4096, 3, (32, 128, 64, 512, 128), (32, 8, 128, 64), 1024, (16, 8, 1376, 4, 3)),
}


def zogevik_named_config(name, layers=0):
    V, d, n, (H, dim, rot, rank, vdim), (AH, G, adim, arot), window, (E, top, ff, groups, keep) = ZOGEVIK_SHAPES[name]
    mlp = experts_config(E, top, ff, groups, keep)
    out, owner = [], None
    for i in range(layers or n):
        if i % 3 != 2:
            out.append(zogevik_latent(H, dim, rot, rank, vdim, window, 10000.0, mlp=mlp))
            continue
        out.append(zogevik_attention(AH, G, adim, adim, arot, window, 10000.0, kv_from=owner, mlp=mlp))
        owner = i if owner is None else None
    return zogevik_config(V, d, out)


def zogevik_named(path, name, seed=0, layers=0):
    """Writes a synthetic model of a named shape; returns its configuration."""
    config = zogevik_named_config(name, layers)
    write(path, config, zogevik_tensors(config, seed=seed, pool=1 << 22))
    return config


def zogevik_tensors(config, seed=0, code=0, pool=0):
    """Random bf16 weights of the shapes a configuration asks for: name -> uint16 array. code > 0: the first `code` entries of
    the residual keep what the embedding put there (the sublayers' norms are 0 on them) and routers read nothing else, so that
    a token's experts do not hang on the last bits of what came before. pool > 0: large matrices are filled from that many
    numbers over and over, each from a place of its own (models of gigabytes)."""
    rng = np.random.default_rng(seed)
    d, V = config["width"], config["vocab"]
    out, base = {}, rng.standard_normal(pool, dtype=np.float32) if pool else None

    def put(name, shape, std, mean=0.0):
        n = int(np.prod(shape))
        if pool and n * 4 > pool:
            bits = to_bf16(base * np.float32(std) + np.float32(mean))
            out[name] = np.resize(np.roll(bits, -int(rng.integers(0, pool))), shape)
            return
        out[name] = to_bf16(rng.standard_normal(shape, dtype=np.float32) * np.float32(std) + np.float32(mean))

    def sublayer_norm(name):
        w = rng.standard_normal(d, dtype=np.float32) * np.float32(0.2) + np.float32(1.0)
        w[:code] = 0.0
        out[name] = to_bf16(w)

    put("embed", (V, d), 1.0)
    put("embed.norm", (d,), 0.2, 1.0)
    for i, layer in enumerate(config["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        H, dim, vdim = m["heads"], m["dim"], m["vdim"]
        sublayer_norm(p + "norm1")
        if layer["type"] == "latent_attention":
            rank, rot = m["kv_rank"], m["rot_dim"]
            put(p + "mix.q", (H * (dim + rot), d), d ** -0.5)
            put(p + "mix.dkv", (rank + rot, d), d ** -0.5)
            put(p + "mix.dkv.norm", (rank,), 0.2, 1.0)
            put(p + "mix.uk", (H * dim, rank), rank ** -0.5)
            put(p + "mix.uv", (H * vdim, rank), rank ** -0.5)
        else:
            G = m["kv_heads"]
            put(p + "mix.q", (H * dim, d), d ** -0.5)
            put(p + "mix.q.norm", (H * dim,), 0.2, 1.0)
            if m.get("kv_from") is None:
                put(p + "mix.k", (G * dim, d), d ** -0.5)
                put(p + "mix.k.norm", (G * dim,), 0.2, 1.0)
                put(p + "mix.v", (G * vdim, d), d ** -0.5)
        put(p + "mix.o", (d, H * vdim), (H * vdim) ** -0.5)
        if not mlp:
            continue
        sublayer_norm(p + "norm2")
        ff = mlp["expert"]["ff"]
        for e in range(mlp["router"]["experts"]):
            put(f"{p}mlp.e{e}.up", (ff, d), d ** -0.5 * 1.5)
            put(f"{p}mlp.e{e}.down", (d, ff), ff ** -0.5)
        n = code or d
        r = np.zeros((mlp["router"]["experts"], d), dtype=np.float32)
        r[:, :n] = rng.standard_normal((r.shape[0], n), dtype=np.float32) * np.float32(n ** -0.5)
        out[p + "mlp.router"] = to_bf16(r)
    put("final.norm", (d,), 0.2, 1.0)
    put("head", (V, d), d ** -0.5)
    return out
