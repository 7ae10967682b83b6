"""Small Metulix models with random weights for the tests: configurations, tensors (bf16-representable, so that the
oracle and the library read the same numbers), a model folder, a session."""
import json
import os

import numpy as np

from emel_cpp_b200 import safetensors as st


def lightning(heads, dim, vdim, decay, ff=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay)},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def attention(heads, kv_heads, dim, vdim, scale, conv=3, rot=(0, 1e4), window=None, keep=0, kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "conv": conv}
    if rot[0]:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    if window is not None:
        m["mask"] = {"size": window, "keep_first": keep}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Metulix", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# sizes that differ everywhere, none a multiple of a tile
ODD = model(72, 101, [
    lightning(3, 24, 40, [0.4, 0.9, 0.995], ff=88),
    attention(6, 2, 20, 28, 0.9, conv=4, rot=(12, 5000.0), window=9, keep=3),
    attention(6, 2, 20, 28, 0.7, conv=2, rot=(12, 5000.0), window=23, keep=0, kv_from=1, ff=50),
    lightning(2, 10, 7, [0.0, 1.0]),
])
# no mask, one key/value head, one tap, unrotated tail, width that needs padding
PLAIN = model(100, 57, [
    attention(4, 1, 34, 50, 0.5, conv=1, rot=(34, 300.0), ff=30),
    lightning(1, 16, 64, [0.97], ff=130),
    attention(5, 5, 16, 24, 1.0, conv=2, window=1, keep=1),
])
# tensor-core sizes
TILED = model(256, 300, [
    attention(8, 2, 128, 128, 0.35, conv=3, rot=(64, 10000.0), window=75, keep=5, ff=384),
    lightning(2, 128, 128, [0.8, 0.999], ff=192),
    attention(8, 2, 128, 128, 0.3, conv=3, rot=(64, 10000.0), window=31, keep=70, kv_from=0),
    attention(12, 4, 64, 32, 0.5, conv=2, rot=(16, 100.0), ff=64),
    lightning(3, 64, 96, [0.5, 0.95, 1.0]),
    lightning(5, 32, 48, [0.99, 0.1, 0.7, 0.98, 0.93]),
])
# many heads, large and uneven groups, value rows wider than a tile
HEADS = model(128, 90, [
    attention(32, 4, 16, 16, 0.6, conv=3, rot=(16, 1000.0), window=40, keep=2),
    attention(40, 8, 16, 8, 0.8, conv=2, rot=(8, 1000.0), window=66, keep=1),
    attention(6, 2, 48, 200, 0.4, conv=4, window=90, keep=80, ff=40),
    lightning(4, 112, 40, [0.9, 0.95, 0.99, 0.3]),
    lightning(2, 144, 24, [0.9, 0.5], ff=24),
])
MODELS = {"heads": HEADS, "odd": ODD, "plain": PLAIN, "tiled": TILED}


def round_bf16(x):
    return st.bf16_to_f32(st.f32_to_bf16(np.asarray(x, np.float32)))


def tensors(cfg, seed):
    g = np.random.Generator(np.random.PCG64(seed))

    def mat(rows, cols, gain=1.0):
        return round_bf16(g.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(n, base=1.0, spread=0.2):
        return round_bf16(base + spread * g.standard_normal(n))

    W, V = cfg["width"], cfg["vocab"]
    t = {"embed": round_bf16(g.standard_normal((V, W))), "final.norm": vec(W), "head": mat(V, W)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, hv = m["heads"], m["heads"] * m["vdim"]
        t[p + "norm1"] = vec(W)
        if layer["type"] == "lightning":
            for n, rows in (("q", H * m["dim"]), ("k", H * m["dim"]), ("v", hv), ("g", hv)):
                t[f"{p}mix.{n}"] = mat(rows, W, 1.5)
            t[p + "mix.norm"] = vec(hv)
        else:
            G = m["kv_heads"]
            parts = {"q": H * m["dim"], "k": G * m["dim"], "v": G * m["vdim"]}
            if m.get("kv_from") is not None:
                parts = {"q": parts["q"]}
            for n, rows in parts.items():
                t[f"{p}mix.{n}"] = mat(rows, W)
                if m["conv"]:
                    t[f"{p}mix.{n}.conv"] = round_bf16(g.standard_normal((rows, m["conv"])) * 0.5 + 0.3)
                if n != "v":
                    t[f"{p}mix.{n}.norm"] = vec(rows)
            t[p + "mix.talk"] = round_bf16(np.eye(H) + 0.3 * g.standard_normal((H, H)))
        t[p + "mix.o"] = mat(W, hv)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            t[p + "norm2"] = vec(W)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(ff, W), mat(ff, W), mat(W, ff)
            t[p + "mlp.gate.b"], t[p + "mlp.up.b"], t[p + "mlp.down.b"] = vec(ff, 0.0), vec(ff, 0.3), vec(W, 0.0)
    return t


def write_folder(path, cfg, t):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    st.write(os.path.join(path, "model.safetensors"), t)
    return str(path)


def as_f64(t):
    return {k: v.astype(np.float64) for k, v in t.items()}


def random_tokens(cfg, n, seed):
    return np.random.Generator(np.random.PCG64(seed)).integers(0, cfg["vocab"], size=n).tolist()


def row_errors(got, want):
    """Root mean square of the centred difference per row, relative to the rows' overall spread."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    spread = np.sqrt(np.mean((want - want.mean(-1, keepdims=True)) ** 2))
    return np.sqrt(np.mean(d * d, axis=-1)) / spread
