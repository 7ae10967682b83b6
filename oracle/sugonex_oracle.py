"""Plain, slow restatement of the Sugonex decoder, one function per mechanism (float64, loops over tokens and heads).
Test infrastructure only: shares no code with the product path.

A model is a config dict ("layers", "loop", "norm", "logit_scale", "logit_softcap", "vocab", "width") and a dict of float
arrays by tensor name.  Every function works on one whole sequence from position 0."""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm(x, weight, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * weight


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def short_conv(u, taps):
    """u [T, channels], taps [channels, n]: causal, the last tap meets the current token."""
    n = taps.shape[1]
    out = np.zeros_like(u)
    for t in range(len(u)):
        for back in range(min(n, t + 1)):
            out[t] += taps[:, n - 1 - back] * u[t - back]
    return out


def rotate_half(x, base, first_pos=0):
    """x [T, ..., d]: dimension i turns with dimension i + d/2."""
    d = x.shape[-1]
    h = d // 2
    y = np.empty_like(x)
    for t in range(len(x)):
        a = (first_pos + t) * float(base) ** (-2.0 * np.arange(h) / d)
        u, v = x[t, ..., :h], x[t, ..., h:]
        y[t, ..., :h] = u * np.cos(a) - v * np.sin(a)
        y[t, ..., h:] = v * np.cos(a) + u * np.sin(a)
    return y


def first_visible(i, window):
    return max(0, i - window + 1) if window else 0


def softmax_attention(q, k, v, scale, window=None):
    """q, k [T, H, d], v [T, H, dv]: each position over itself and the (window - 1, or all) positions before it."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for i in range(T):
        lo = first_visible(i, window)
        for h in range(H):
            s = k[lo:i + 1, h] @ q[i, h] * scale
            e = np.exp(s - s.max())
            out[i, h] = (e / e.sum()) @ v[lo:i + 1, h]
    return out


def latent_mixer(h, w, p, m, eps, gated):
    """Keys and values of all heads come from one normed latent per token; a rotated key part is shared by the heads."""
    T, H, d, r, rank = len(h), m["heads"], m["dim"], m.get("rot_dim") or 0, m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :rank], w[p + "dkv.norm"], eps)
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    if r:
        q = np.concatenate([q[..., :d], rotate_half(q[..., d:], m["rot"]["base"])], axis=-1)
        shared = rotate_half(down[:, rank:], m["rot"]["base"])
        k = np.concatenate([k, np.repeat(shared[:, None], H, axis=1)], axis=-1)
    o = softmax_attention(q, k, v, m["scale"], (m.get("mask") or {}).get("size")).reshape(T, -1)
    if gated:
        o = o * sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def delta_rule(q, k, v, beta, g, state=None):
    """q, k [T, H, d] (one per head), v [T, H, dv], beta and g [T, H] -> outputs and the final state [H, d, dv]."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + np.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def delta_decay(a, a_log, dt_bias):
    return np.exp(-np.exp(a_log) * softplus(a + dt_bias))


def delta_inputs(h, w, p, m):
    T, H, G, d, dv = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    parts = {n: silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"])) for n in "qkv"}
    q, k = (unit(parts[n].reshape(T, G, d)) for n in "qk")
    q = q * d ** -0.5
    q, k = (np.repeat(x, H // G, axis=1) for x in (q, k))
    beta = sigmoid(h @ w[p + "b"].T)
    g = delta_decay(h @ w[p + "a"].T, w[p + "A_log"], w[p + "dt_bias"])
    return q, k, parts["v"].reshape(T, H, dv), beta, g


def delta_mixer(h, w, p, m, eps):
    T, H, dv = len(h), m["heads"], m["vdim"]
    o, _ = delta_rule(*delta_inputs(h, w, p, m))
    o = rms_norm(o, w[p + "norm"], eps) * silu(h @ w[p + "g"].T).reshape(T, H, dv)
    return o.reshape(T, -1) @ w[p + "o"].T


def gated_mlp(h, w, p):
    return (gelu_tanh(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def layer_order(cfg):
    """(layer, pass that starts ahead of it or None) for every layer run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        out += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return out + [(i, None) for i in range(loop["stop"], n)]


def layer(cfg, w, i, x):
    eps, l, p = cfg["norm"]["eps"], cfg["layers"][i], f"l{i}."
    h = rms_norm(x, 1.0 + w[p + "norm1"], eps)
    if l["type"] == "delta":
        y = delta_mixer(h, w, p + "mix.", l["mixer"], eps)
    else:
        y = latent_mixer(h, w, p + "mix.", l["mixer"], eps, gated=l["type"] == "latent_attention")
    if l.get("mlp"):
        y = y + gated_mlp(rms_norm(x, 1.0 + w[p + "norm2"], eps), w, p + "mlp.")
    return x + y


def residual_streams(cfg, w, tokens):
    """The residual stream after every layer run, [runs, T, width]."""
    x = w["embed"][np.asarray(tokens)]
    out = []
    for i, t in layer_order(cfg):
        if t is not None:
            x = x + w["loop.step"][t]
        x = layer(cfg, w, i, x)
        out.append(x)
    return np.stack(out)


def head(cfg, w, x):
    z = rms_norm(x, 1.0 + w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z


def logits(cfg, w, tokens):
    return head(cfg, w, residual_streams(cfg, w, tokens)[-1])
