"""Small Sugonex models with random weights for the tests: configurations and tensors (bf16-representable, so that the oracle
and the library read the same numbers).  Folders, tokens and error measures are those of the Metulix tests."""
import numpy as np

from tests.metulix_models import as_f64, random_tokens, round_bf16, row_errors, write_folder  # noqa: F401


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot, vdim, rank, scale, base=1e4, ff=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"dims": rot, "base": base}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def windowed(heads, dim, vdim, rank, scale, window, ff=None):
    return {"type": "latent_attention_2",
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale, "mask": {"size": window}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def model(width, vocab, layers, loop=None, eps=1e-5, scale=0.7, cap=20.0):
    m = {"architecture": "Sugonex", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "logit_scale": scale,
         "logit_softcap": cap}
    if loop:
        m["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return m


# sizes that differ everywhere, none a multiple of a tile; one layer looped
ODD = model(76, 103, [
    windowed(3, 22, 30, 27, 0.9, 9, ff=90),
    delta(6, 2, 20, 28, 3, ff=50),
    latent(5, 18, 6, 26, 35, 0.7, base=700.0, ff=34),
    delta(3, 3, 9, 7, 5),
], loop=(1, 2, 4))
# one tap, one head, a window of one, no feed-forwards, the whole stack looped, no cap
PLAIN = model(100, 57, [
    delta(1, 1, 33, 17, 1),
    latent(1, 40, 2, 10, 12, 0.5),
    windowed(2, 8, 50, 60, 1.0, 1),
], loop=(0, 3, 2), cap=None, scale=1.0)
# tensor-core sizes, loop at the end
TILED = model(256, 300, [
    latent(4, 64, 32, 96, 160, 0.2, base=5e4, ff=384),
    delta(8, 2, 128, 128, 4, ff=320),
    windowed(12, 48, 32, 96, 0.3, 70, ff=64),
    delta(3, 3, 48, 80, 2, ff=128),
    latent(2, 128, 64, 128, 512, 0.15, base=1e4),
], loop=(3, 5, 2))
# many heads, a wide latent, value rows wider than a tile, a loop of one pass
HEADS = model(128, 90, [
    latent(20, 16, 8, 16, 24, 0.6, ff=40),
    delta(16, 4, 16, 24, 4, ff=56),
    windowed(9, 32, 136, 600, 0.4, 33),
    delta(2, 1, 144, 200, 3, ff=24),
    delta(4, 2, 64, 32, 4),
], loop=(2, 4, 1))
MODELS = {"heads": HEADS, "odd": ODD, "plain": PLAIN, "tiled": TILED}


def tensors(cfg, seed):
    g = np.random.Generator(np.random.PCG64(seed))

    def mat(rows, cols, gain=1.0):
        return round_bf16(g.standard_normal((rows, cols)) * gain / np.sqrt(cols))

    def vec(n, base=1.0, spread=0.2):
        return round_bf16(base + spread * g.standard_normal(n))

    W, V = cfg["width"], cfg["vocab"]
    t = {"embed": round_bf16(g.standard_normal((V, W))), "final.norm": vec(W, 0.0)}
    if cfg.get("loop"):
        t["loop.step"] = round_bf16(0.5 * g.standard_normal((cfg["loop"]["times"], W)))
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        H, hv = m["heads"], m["heads"] * m["vdim"]
        t[p + "norm1"] = vec(W, 0.0)
        if layer["type"] == "delta":
            G = m["kv_heads"]
            for n, rows in (("q", G * m["dim"]), ("k", G * m["dim"]), ("v", hv)):
                t[f"{p}mix.{n}"] = mat(rows, W, 1.5)
                t[f"{p}mix.{n}.conv"] = round_bf16(g.standard_normal((rows, m["conv"])) * 0.5 + 0.3)
            t[p + "mix.g"], t[p + "mix.b"], t[p + "mix.a"] = mat(hv, W), mat(H, W, 1.5), mat(H, W)
            # decays from about 0.3 to 0.999 a token
            t[p + "mix.A_log"] = round_bf16(np.linspace(-4.0, 0.5, H) + 0.1 * g.standard_normal(H))
            t[p + "mix.dt_bias"] = vec(H, -0.5, 0.5)
            t[p + "mix.norm"] = vec(m["vdim"])
        else:
            rot = m.get("rot_dim") or 0
            t[p + "mix.q"] = mat(H * (m["dim"] + rot), W, 1.5)
            t[p + "mix.dkv"] = mat(m["kv_rank"] + rot, W)
            t[p + "mix.dkv.norm"] = vec(m["kv_rank"])
            t[p + "mix.uk"], t[p + "mix.uv"] = mat(H * m["dim"], m["kv_rank"], 1.5), mat(hv, m["kv_rank"])
            if layer["type"] == "latent_attention":
                t[p + "mix.g"] = mat(hv, W)
        t[p + "mix.o"] = mat(W, hv)
        if layer.get("mlp"):
            ff = layer["mlp"]["ff"]
            t[p + "norm2"] = vec(W, 0.0)
            t[p + "mlp.gate"], t[p + "mlp.up"], t[p + "mlp.down"] = mat(ff, W), mat(ff, W), mat(W, ff)
    return t
