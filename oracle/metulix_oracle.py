"""Plain, slow restatement of the Metulix decoder, one function per mechanism (float64, loops over
tokens and heads).  Test infrastructure only: shares no code with the product path.

A model is a config dict ("layers", "norm", "vocab", "width") and a dict of float arrays by tensor
name.  Every function works on one whole sequence from position 0."""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, weight=None, eps=1e-6):
    y = x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def layer_norm(x, weight, eps):
    d = x - np.mean(x, axis=-1, keepdims=True)
    return d / np.sqrt(np.mean(d * d, axis=-1, keepdims=True) + eps) * weight


def short_conv(u, taps):
    """u [T, channels], taps [channels, n]: causal, tap n-1 meets the current token."""
    n = taps.shape[1]
    out = np.zeros_like(u)
    for t in range(len(u)):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] += taps[:, j] * u[src]
    return out


def rotate(x, dims, base, first_pos=0):
    """x [T, heads, d]: adjacent pairs of the first `dims` dimensions of every head."""
    y = x.copy()
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        a = (first_pos + np.arange(len(x))) * f
        c, s = np.cos(a)[:, None], np.sin(a)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * c - v * s
        y[:, :, 2 * i + 1] = v * c + u * s
    return y


def visible(i, j, mask):
    if j > i:
        return False
    if not mask:
        return True
    return i - j < mask["size"] or j < mask.get("keep_first", 0)


def talking_attention(q, k, v, scale, mask, talk):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: softmax per head over the visible keys, heads' weights
    mixed by talk [H, H], head h then weighs the values of its own key/value head."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        js = [j for j in range(i + 1) if visible(i, j, mask)]
        w = np.zeros((H, len(js)))
        for h in range(H):
            s = k[js, h // (H // G)] @ q[i, h] * scale
            e = np.exp(s - s.max())
            w[h] = e / e.sum()
        w = talk @ w
        for h in range(H):
            out[i, h] = w[h] @ v[js, h // (H // G)]
    return out


def lightning(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, dv] -> outputs and the final state [H, d, dv]."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def gated_mlp(x, w, p):
    g = x @ w[p + "gate"].T + w[p + "gate.b"]
    u = x @ w[p + "up"].T + w[p + "up.b"]
    return (silu(g) * u) @ w[p + "down"].T + w[p + "down.b"]


def lightning_mixer(x, w, p, m, eps):
    T, H = len(x), m["heads"]
    q = silu(x @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = silu(x @ w[p + "k"].T).reshape(T, H, m["dim"])
    v = silu(x @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o, _ = lightning(q, k, v, m["decay"])
    o = rms_norm(o.reshape(T, -1), w[p + "norm"], eps) * sigmoid(x @ w[p + "g"].T)
    return o @ w[p + "o"].T


def attention_mixer(x, w, p, m, eps, lent):
    """lent: layer index -> (keys as cached, values after the convolution) of the layers before; returns the output and
    this layer's own entry (None for a layer that borrows).  A mechanism whose tensors are missing is left out."""
    T, H, G = len(x), m["heads"], m["kv_heads"]
    rot = m.get("rot") or {"dims": 0, "base": 1.0}

    def projected(name):
        u = x @ w[p + name].T
        return short_conv(u, w[p + name + ".conv"]) if p + name + ".conv" in w else u

    def normed(u, name):
        return rms_norm(u, w[p + name + ".norm"], eps) if p + name + ".norm" in w else u

    q = rotate(normed(projected("q"), "q").reshape(T, H, m["dim"]), rot["dims"], rot["base"])
    own = None
    if m.get("kv_from") is None:
        k = rotate(normed(projected("k"), "k").reshape(T, G, m["dim"]), rot["dims"], rot["base"])
        raw = projected("v").reshape(T, G, m["vdim"])
        own = (k, raw)
    else:
        k, raw = lent[m["kv_from"]]
    v = rms_norm(raw, None, eps) if m.get("norm_v", True) else raw
    talk = w[p + "talk"] if p + "talk" in w else np.eye(H)
    o = talking_attention(q, k, v, m["scale"], m.get("mask"), talk)
    return o.reshape(T, -1) @ w[p + "o"].T, own


def residual_streams(cfg, w, tokens):
    """The residual stream after every layer, [layers, T, width]."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    lent, out = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        if layer["type"] == "lightning":
            y = lightning_mixer(x, w, p + "mix.", layer["mixer"], eps)
        else:
            y, own = attention_mixer(x, w, p + "mix.", layer["mixer"], eps, lent)
            if own is not None:
                lent[i] = own
        x = x + layer_norm(y, w[p + "norm1"], eps)
        if layer.get("mlp"):
            x = x + layer_norm(gated_mlp(x, w, p + "mlp."), w[p + "norm2"], eps)
        out.append(x)
    return np.stack(out)


def logits(cfg, w, tokens):
    x = residual_streams(cfg, w, tokens)[-1]
    return layer_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].T
