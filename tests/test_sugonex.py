"""Sugonex without a GPU: the oracle's mechanisms against independent closed forms, that planted mistakes show, the configuration
reader and its checks, what the loader binds, and the registry."""
import copy

import numpy as np
import pytest

import emel_cpp_b200 as eb
from emel_cpp_b200 import layered as ly
from emel_cpp_b200 import models, safetensors as st
from emel_cpp_b200 import sugonex as sx
from oracle import sugonex_oracle as so
from tests import sugonex_models as sm


def test_short_convolution_is_causal_and_starts_from_zero():
    g = np.random.default_rng(1)
    u, w = g.standard_normal((9, 4)), g.standard_normal((4, 3))
    assert np.allclose(so.short_conv(u, w), np.stack([np.convolve(u[:, c], w[c, ::-1])[:9] for c in range(4)], 1))
    assert np.allclose(so.short_conv(u, w[:, 2:]), u * w[:, 2])


def test_rotation_of_halves_keeps_relative_angles():
    g = np.random.default_rng(2)
    q, k = g.standard_normal((1, 3, 10)), g.standard_normal((1, 3, 10))
    a = [float((so.rotate_half(q, 50.0, p + 4) * so.rotate_half(k, 50.0, p)).sum()) for p in (0, 7, 90)]
    assert np.allclose(a, a[0])
    # as complex numbers: first half + i second half, turned by position * base^(-2 i / d)
    z = (q[..., :5] + 1j * q[..., 5:]) * np.exp(3j * 50.0 ** (-np.arange(5) / 5.0))
    r = so.rotate_half(q, 50.0, 3)
    assert np.allclose(r[..., :5], z.real) and np.allclose(r[..., 5:], z.imag)


def test_windows():
    assert [so.first_visible(i, 3) for i in range(6)] == [0, 0, 0, 1, 2, 3]
    assert [so.first_visible(i, None) for i in (0, 5)] == [0, 0] and so.first_visible(7, 1) == 7
    g = np.random.default_rng(3)
    q, k, v = g.standard_normal((8, 2, 5)), g.standard_normal((8, 2, 5)), g.standard_normal((8, 2, 3))
    got = so.softmax_attention(q, k, v, 0.4, 3)
    for h in range(2):
        s = q[:, h] @ k[:, h].T * 0.4
        s = np.where(np.tril(np.ones((8, 8))) * np.triu(np.ones((8, 8)), -2) > 0, s, -np.inf)
        p = np.exp(s - s.max(1, keepdims=True))
        assert np.allclose(got[:, h], p / p.sum(1, keepdims=True) @ v[:, h])


def test_latent_keys_can_be_absorbed_by_the_query():
    """Scores against the latents themselves, with the key rows applied to the query, are the same scores."""
    g = np.random.default_rng(4)
    q, U, c = g.standard_normal(6), g.standard_normal((6, 9)), g.standard_normal((5, 9))
    assert np.allclose((c @ U.T) @ q, c @ (U.T @ q))


def test_delta_rule_in_closed_form():
    g = np.random.default_rng(5)
    T, d, dv = 13, 5, 3
    q, k, v = so.unit(g.standard_normal((T, 1, d))), so.unit(g.standard_normal((T, 1, d))), g.standard_normal((T, 1, dv))
    beta, decay = g.uniform(0, 1, (T, 1)), g.uniform(0.5, 1, (T, 1))
    o, S = so.delta_rule(q, k, v, beta, decay)
    # (I + A) U = beta v with A_ij = beta_i decay(j+1..i) k_i.k_j below the diagonal
    G = np.cumsum(np.log(decay[:, 0]))
    D = np.tril(np.exp(G[:, None] - G[None]))
    A = np.tril(beta * D * (k[:, 0] @ k[:, 0].T), -1)
    U = np.linalg.solve(np.eye(T) + A, beta * v[:, 0])
    assert np.allclose(o[:, 0], (D * (q[:, 0] @ k[:, 0].T)) @ U)
    assert np.allclose(S[0], (k[:, 0] * D[-1][:, None]).T @ U)
    head, S1 = so.delta_rule(q[:6], k[:6], v[:6], beta[:6], decay[:6])
    tail, S2 = so.delta_rule(q[6:], k[6:], v[6:], beta[6:], decay[6:], S1)
    assert np.allclose(np.concatenate([head, tail]), o) and np.allclose(S, S2)


def test_delta_rule_overwrites_what_a_key_held():
    """With step size 1 and no decay, writing under a key replaces its value, and the same token reads it back."""
    k = np.zeros((3, 1, 4))
    k[0, 0, 1] = k[2, 0, 1] = k[1, 0, 2] = 1.0
    v = np.arange(1.0, 7.0).reshape(3, 1, 2)
    o, S = so.delta_rule(k, k, v, np.ones((3, 1)), np.ones((3, 1)))
    assert np.allclose(o, v) and np.allclose(S[0, 1], v[2, 0]) and np.allclose(S[0, 2], v[1, 0])


def test_heads_share_queries_and_keys_in_order():
    m = {"heads": 6, "kv_heads": 2, "dim": 4, "vdim": 3}
    g = np.random.default_rng(6)
    w = {"q": g.standard_normal((8, 5)), "k": g.standard_normal((8, 5)), "v": g.standard_normal((18, 5)), "b": g.standard_normal((6, 5)),
         "a": g.standard_normal((6, 5)), "A_log": g.standard_normal(6), "dt_bias": g.standard_normal(6)}
    for n, r in (("q", 8), ("k", 8), ("v", 18)):
        w[n + ".conv"] = g.standard_normal((r, 2))
    q, k, v, beta, decay = so.delta_inputs(g.standard_normal((7, 5)), w, "", m)
    assert q.shape == (7, 6, 4) and v.shape == (7, 6, 3)
    for x in (q, k):
        assert np.allclose(x[:, 0], x[:, 2]) and np.allclose(x[:, 3], x[:, 5]) and not np.allclose(x[:, 2], x[:, 3])
    assert np.allclose((k ** 2).sum(-1), 1, atol=1e-4) and np.allclose((q ** 2).sum(-1), 0.25, atol=1e-4)
    assert (0 < decay).all() and (decay < 1).all() and (0 < beta).all() and (beta < 1).all()


def test_gelu_and_softplus():
    z = np.linspace(-6, 6, 25)
    y = np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3)
    assert np.allclose(so.gelu_tanh(z), z * so.sigmoid(2 * y)) and np.allclose(so.softplus(z), np.log1p(np.exp(z)))


def test_order_of_layers():
    assert so.layer_order(sm.ODD) == [(0, None), (1, 0), (1, 1), (1, 2), (1, 3), (2, None), (3, None)]
    assert so.layer_order(sm.TILED) == [(0, None), (1, None), (2, None), (3, 0), (4, None), (3, 1), (4, None)]
    assert so.layer_order(sm.PLAIN)[:3] == [(0, 0), (1, None), (2, None)]


def _mistakes(cfg):
    """Configurations with one thing wrong."""
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        if m.get("mask"):
            for by in (1, -1):
                if m["mask"]["size"] + by >= 1:
                    c = copy.deepcopy(cfg)
                    c["layers"][i]["mixer"]["mask"]["size"] += by
                    yield f"layer {i} window {by:+d}", c
        for path, f in ((("rot", "base"), 1.5), (("scale",), 1.05)):
            # one pair turns by one radian per token whatever the base, and one visible key has all the weight whatever its score
            if path[0] in m and m.get("rot_dim") != 2 and (m.get("mask") or {}).get("size") != 1:
                c = copy.deepcopy(cfg)
                x = c["layers"][i]["mixer"]
                for k in path[:-1]:
                    x = x[k]
                x[path[-1]] *= f
                yield f"layer {i} {path}", c
    for key, f in (("logit_scale", 1.02), ("logit_softcap", 0.9)):
        if cfg.get(key):
            c = copy.deepcopy(cfg)
            c[key] *= f
            yield key, c
    if cfg.get("loop") and cfg["loop"]["times"] > 1:
        c = copy.deepcopy(cfg)
        c["loop"]["times"] -= 1
        yield "passes", c


@pytest.mark.parametrize("name", ["odd", "plain", "tiled"])
def test_planted_mistakes_show(name):
    """The weights make every window edge, angle and constant visible well above the tolerance of the GPU tests."""
    cfg = sm.MODELS[name]
    w, toks = sm.as_f64(sm.tensors(cfg, 5)), sm.random_tokens(cfg, 110, 6)
    good = so.logits(cfg, w, toks)
    for what, bad in _mistakes(cfg):
        e = sm.row_errors(so.logits(bad, w, toks), good)
        assert e.max() > 2e-3, (what, e.max())
    for part in ("conv", "dkv.norm", "mix.g", "A_log", "dt_bias", "norm1", "loop.step"):
        bad = {k: (v + 0.1 if part in k else v) for k, v in w.items()}
        if any(part in k for k in w):
            assert sm.row_errors(so.logits(cfg, bad, toks), good).max() > 2e-3, part


def test_configuration_reader():
    layers = sx.layer_configs(sm.ODD)
    assert [l.mixer for l in layers] == [ly.MIXER_LATENT, ly.MIXER_DELTA, ly.MIXER_LATENT, ly.MIXER_DELTA]
    a, b, c = layers[0], layers[1], layers[2]
    assert (a.n_head, a.key_dim, a.value_dim, a.kv_rank, a.rope_dim, a.window, a.out_gate, a.n_ff) == (3, 22, 30, 27, 0, 9, 0, 90)
    assert (b.n_head, b.n_head_kv, b.key_dim, b.value_dim, b.conv_taps, b.n_ff, b.ff_act) == (6, 2, 20, 28, 3, 50, ly.FF_GELU_TANH)
    assert (c.rope_dim, c.rope_half, c.out_gate, c.window, c.kv_rank) == (6, 1, 1, 0, 35) and c.rope_freq_base == 700.0
    assert [ly.in_rows(l) for l in layers] == [3 * 22 + 27, 2 * 40 + 2 * 168 + 12, 5 * (24 + 26) + 41, 2 * 27 + 2 * 21 + 6]
    s = sx.stack_config(sm.ODD)
    assert (s.arrangement, s.norm, s.loop_start, s.loop_stop, s.loop_times, s.loop_step) == (ly.STACK_PARALLEL, ly.NORM_RMS, 1, 2, 4, 1)
    assert (round(s.logit_scale, 6), s.logit_softcap) == (0.7, 20.0)
    plain = {k: v for k, v in sm.PLAIN.items() if k not in ("loop", "logit_scale", "logit_softcap")}
    s = sx.stack_config(plain)
    assert (s.loop_times, s.loop_step, s.logit_scale, s.logit_softcap) == (0, 0, 1.0, 0.0)
    for change in (lambda c: c["layers"][0].update(type="conv"), lambda c: c["layers"][0]["mlp"].update(kind="experts"),
                   lambda c: c["layers"][2]["mixer"]["rot"].update(dims=4)):
        bad = copy.deepcopy(sm.ODD)
        change(bad)
        with pytest.raises(ValueError):
            sx.layer_configs(bad)


def test_stack_checks():
    def check(change=None, **cfg):
        base = dict(n_layer=2, n_embd=64, n_vocab=10, n_ctx=32, eps=1e-6)
        base.update(cfg)
        a = ly.latent_layer(4, 16, 16, 24, 0.25, rope_dim=8, window=5, n_ff=8)
        b = ly.delta_layer(4, 2, 16, 16, 3)
        s = ly.stack(ly.STACK_PARALLEL, ly.NORM_RMS, loop=(0, 2, 3), loop_step=True, logit_scale=0.5, logit_softcap=3.0)
        if change:
            change(a, b, s)
        return ly.check_layers(ly.config(**base), [a, b], s)

    assert check() == eb.OK and check(n_embd=0) == eb.INVALID_REQUEST
    for field, bad in (("kv_rank", 0), ("rope_dim", 7), ("rope_dim", -2), ("window", -1), ("n_head", 0), ("ff_act", 9), ("mixer", 7), ("rope_freq_base", 0.0)):
        assert check(lambda a, b, s: setattr(a, field, bad)) == eb.INVALID_REQUEST, (field, bad)
    for field, bad in (("n_head_kv", 3), ("n_head_kv", 0), ("conv_taps", 0), ("value_dim", 0), ("key_dim", 2000)):
        assert check(lambda a, b, s: setattr(b, field, bad)) == eb.INVALID_REQUEST, (field, bad)
    for field, bad in (("arrangement", 2), ("norm", 2), ("loop_stop", 3), ("loop_stop", 0), ("loop_start", -1), ("loop_times", -1), ("loop_times", 0),
                       ("logit_softcap", -1.0), ("logit_scale", float("nan"))):
        assert check(lambda a, b, s: setattr(s, field, bad)) == eb.INVALID_REQUEST, (field, bad)


class Recorder:
    """Stands for a session: what is bound, by layer and role."""

    def __init__(self):
        self.bound = {}

    def load_matrix(self, layer, role, bits, also=()):
        for key in [(layer, role), *also]:
            self.bound[key] = st.bf16_to_f32(np.asarray(bits))
        return True

    def load_vector(self, layer, role, values):
        self.bound[(layer, role)] = np.asarray(values)
        return True

    def close(self):
        pass


def test_loader_stacks_and_shifts(tmp_path, monkeypatch):
    cfg, t = sm.ODD, sm.tensors(sm.ODD, 3)
    sm.write_folder(tmp_path / "m", cfg, t)
    rec = Recorder()

    def session(backend, config, layers, float32, stack):
        rec.layers, rec.stack = layers, stack
        return rec
    monkeypatch.setattr(ly, "Session", session)
    assert models.load(None, str(tmp_path / "m"), n_ctx=64) is rec
    from emel_cpp_b200 import llama as el
    b = rec.bound
    assert np.array_equal(b[(-1, el.TOKEN_EMBD)], t["embed"]) and np.array_equal(b[(-1, el.OUTPUT)], t["embed"])
    assert np.array_equal(b[(-1, el.OUTPUT_NORM)], np.float32(1) + t["final.norm"]) and np.array_equal(b[(-1, ly.LOOP_STEP)], t["loop.step"])
    assert np.array_equal(b[(1, ly.MIX_IN)], np.concatenate([t[f"l1.mix.{n}"] for n in ("q", "k", "v", "g", "b", "a")]))
    assert np.array_equal(b[(2, ly.MIX_IN)], np.concatenate([t[f"l2.mix.{n}"] for n in ("q", "g", "dkv")]))
    assert np.array_equal(b[(0, ly.MIX_IN)], np.concatenate([t["l0.mix.q"], t["l0.mix.dkv"]]))
    out = b[(1, ly.LAYER_OUT)]
    od = 6 * 28
    assert out.shape == (76, 168 + 50) and np.array_equal(out[:, :od], t["l1.mix.o"]) and np.array_equal(out[:, 168:], t["l1.mlp.down"])
    out = b[(0, ly.LAYER_OUT)]
    assert out.shape == (76, 96 + 90) and np.array_equal(out[:, :90], t["l0.mix.o"]) and not out[:, 90:96].any()
    assert (3, ly.LAYER_OUT) not in b and np.array_equal(b[(3, el.ATTN_OUT)], t["l3.mix.o"])
    for i, l in enumerate(rec.layers):
        assert b[(i, ly.MIX_IN)].shape == (ly.in_rows(l), 76)


def test_registry():
    assert {"Metulix", "Sugonex", "llama"} <= set(models.ARCHITECTURES)
