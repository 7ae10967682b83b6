"""Metulix without a GPU: the oracle's mechanisms against independent closed forms, that planted mistakes show, the
configuration reader and its checks, the safetensors reader, the registry, and the trace replay's bookkeeping."""
import copy
import io
import json

import numpy as np
import pytest

import emel_cpp_b200 as eb
from emel_cpp_b200 import layered as ly
from emel_cpp_b200 import metulix as mx
from emel_cpp_b200 import models, safetensors as st, trace
from oracle import metulix_oracle as mo
from tests import metulix_models as mm


def test_short_convolution_is_causal_and_starts_from_zero():
    g = np.random.default_rng(1)
    u, w = g.standard_normal((9, 4)), g.standard_normal((4, 3))
    want = np.stack([np.convolve(u[:, c], w[c, ::-1])[:9] for c in range(4)], 1)
    assert np.allclose(mo.short_conv(u, w), want)


def test_rotation_keeps_relative_angles_and_the_tail():
    g = np.random.default_rng(2)
    q, k = g.standard_normal((1, 1, 10)), g.standard_normal((1, 1, 10))
    a = [float((mo.rotate(q, 6, 50.0, p + 4) * mo.rotate(k, 6, 50.0, p)).sum()) for p in (0, 7, 90)]
    assert np.allclose(a, a[0])
    assert np.array_equal(mo.rotate(q, 6, 50.0, 3)[..., 6:], q[..., 6:])


def test_lightning_state_is_the_decayed_sum():
    g = np.random.default_rng(3)
    q, k, v = (g.standard_normal((12, 2, d)) for d in (5, 5, 3))
    decay = [0.7, 0.95]
    o, S = mo.lightning(q, k, v, decay)
    for h in range(2):
        lam = np.array([[decay[h] ** (i - j) if j <= i else 0.0 for j in range(12)] for i in range(12)])
        assert np.allclose(o[:, h], ((q[:, h] @ k[:, h].T) * lam) @ v[:, h])
    head, S1 = mo.lightning(q[:5], k[:5], v[:5], decay)
    tail, S2 = mo.lightning(q[5:], k[5:], v[5:], decay, S1)
    assert np.allclose(np.concatenate([head, tail]), o) and np.allclose(S, S2)


def test_window_keeps_the_first_tokens():
    mask = {"size": 3, "keep_first": 2}
    assert [j for j in range(12) if mo.visible(9, j, mask)] == [0, 1, 7, 8, 9]
    assert [j for j in range(12) if mo.visible(3, j, mask)] == [0, 1, 2, 3]
    assert [j for j in range(12) if mo.visible(5, j, None)] == [0, 1, 2, 3, 4, 5]


def test_heads_are_mixed_after_the_softmax():
    g = np.random.default_rng(4)
    q, k, v = g.standard_normal((6, 4, 8)), g.standard_normal((6, 2, 8)), g.standard_normal((6, 2, 3))
    T = g.standard_normal((4, 4))
    mixed = mo.talking_attention(q, k, v, 0.4, None, T)
    # head g's weights applied to each value head, then combined
    for h in range(4):
        want = 0.0
        for gg in range(4):
            kk = np.repeat(k, 2, axis=1)[:, gg:gg + 1]
            vv = v[:, h // 2:h // 2 + 1]
            want = want + T[h, gg] * mo.talking_attention(q[:, gg:gg + 1], kk, vv, 0.4, None, np.eye(1))[:, 0]
        assert np.allclose(mixed[:, h], want)


def _mistakes(cfg):
    """Configurations with one thing wrong."""
    for i, layer in enumerate(cfg["layers"]):
        m = layer["mixer"]
        if layer["type"] == "lightning":
            c = copy.deepcopy(cfg)
            c["layers"][i]["mixer"]["decay"] = [d * 0.98 for d in m["decay"]]
            yield f"layer {i} decay", c
            continue
        if m.get("mask"):
            for key, by in (("size", 1), ("size", -1), ("keep_first", 1), ("keep_first", -1)):
                if m["mask"][key] + by >= (1 if key == "size" else 0):
                    c = copy.deepcopy(cfg)
                    c["layers"][i]["mixer"]["mask"][key] += by
                    yield f"layer {i} {key} {by:+d}", c
        if m.get("rot"):
            c = copy.deepcopy(cfg)
            c["layers"][i]["mixer"]["rot"]["base"] *= 1.3
            yield f"layer {i} base", c


@pytest.mark.parametrize("name", ["odd", "plain"])
def test_planted_mistakes_show(name):
    """The weights make every mask edge, decay and angle visible well above the tolerance of the GPU tests."""
    cfg = mm.MODELS[name]
    w, toks = mm.as_f64(mm.tensors(cfg, 5)), mm.random_tokens(cfg, 60, 6)
    good = mo.logits(cfg, w, toks)
    for what, bad in _mistakes(cfg):
        e = mm.row_errors(mo.logits(bad, w, toks), good)
        assert e.max() > 2e-3, (what, e.max())
    for drop in ("talk", "conv"):
        bad = {k: v for k, v in w.items() if not k.endswith(drop)}
        assert mm.row_errors(mo.logits(cfg, bad, toks), good).max() > 2e-2, drop


def test_configuration_reader():
    layers = mx.layer_configs(mm.ODD)
    assert [l.mixer for l in layers] == [ly.MIXER_LINEAR, ly.MIXER_ATTENTION, ly.MIXER_ATTENTION, ly.MIXER_LINEAR]
    a = layers[1]
    assert (a.n_head, a.n_head_kv, a.key_dim, a.value_dim, a.conv_taps, a.rope_dim, a.window, a.keep_first, a.kv_from, a.n_ff) == \
        (6, 2, 20, 28, 4, 12, 9, 3, -1, 0)
    assert layers[2].kv_from == 1 and layers[0].n_ff == 88
    assert [ly.in_rows(l) for l in layers] == [3 * 2 * 64, 6 * 20 + 2 * 48, 120, 2 * 2 * 17]
    assert [layers[0].decay[i] for i in range(3)] == [np.float32(d) for d in (0.4, 0.9, 0.995)]
    bad = copy.deepcopy(mm.ODD)
    bad["layers"][0]["type"] = "conv"
    with pytest.raises(ValueError):
        mx.layer_configs(bad)


def test_layer_checks():
    def check(change=None, **cfg):
        base = dict(n_layer=2, n_embd=64, n_vocab=10, n_ctx=32, eps=1e-6)
        base.update(cfg)
        a = ly.attention_layer(4, 2, 16, 16, 0.25, conv_taps=3, rope_dim=8, window=5, keep_first=1, n_ff=8)
        b = ly.attention_layer(4, 2, 16, 16, 0.25, conv_taps=3, rope_dim=8, kv_from=0)
        if change:
            change(a, b)
        return ly.check_layers(ly.config(**base), [a, b])

    assert check() == eb.OK
    assert check(n_embd=0) == eb.INVALID_REQUEST and check(n_ctx=0) == eb.INVALID_REQUEST
    for change in (lambda a, b: setattr(a, "n_head_kv", 3), lambda a, b: setattr(a, "rope_dim", 18), lambda a, b: setattr(a, "rope_dim", 7),
                   lambda a, b: setattr(b, "kv_from", 1), lambda a, b: setattr(b, "kv_from", -2), lambda a, b: setattr(a, "kv_from", 0),
                   lambda a, b: setattr(b, "key_dim", 8), lambda a, b: setattr(b, "norm_v", 0), lambda a, b: setattr(a, "mixer", 7),
                   lambda a, b: setattr(a, "window", -1), lambda a, b: setattr(a, "mixer", ly.MIXER_LINEAR)):
        assert check(change) == eb.INVALID_REQUEST


def test_safetensors_round_trip(tmp_path):
    x = np.array([[1.0, -2.5, 3.14159], [0.0, 1e-30, 65504.0]], np.float32)
    ids = np.arange(4, dtype=np.int32)
    st.write(str(tmp_path / "m.safetensors"), {"x": x, "ids": ids})
    f = st.File(str(tmp_path / "m.safetensors"))
    assert sorted(f.names()) == ["ids", "x"] and f.shape("x") == (2, 3) and f.dtype("ids") == "I32"
    assert np.array_equal(f.array("ids"), ids)
    assert np.allclose(f.f32("x"), x, rtol=2 ** -8) and np.array_equal(st.bf16_to_f32(f.bf16("x")), f.f32("x"))


def test_registry(tmp_path):
    path = mm.write_folder(tmp_path / "m", mm.ODD, {"embed": np.zeros((2, 2), np.float32)})
    assert models.architecture(path) == "Metulix" and {"Metulix", "llama"} <= set(models.ARCHITECTURES)
    (tmp_path / "m" / "config.json").write_text(json.dumps({"architecture": "Nothing"}))
    with pytest.raises(ValueError):
        models.load(None, path)


class FakeSession:
    """Counts tokens per sequence; the logits row of a place is [sequence, position, token]."""
    last_error = 0

    def __init__(self):
        self.seq, self.calls = 0, []

    def select_sequence(self, s):
        self.seq = s
        return True

    def prefill_logits(self, tokens, start, want):
        self.calls.append((self.seq, start, len(tokens)))
        return np.array([[self.seq, start + w, tokens[w]] for w in want], np.float32).reshape(len(want), 3)


def test_trace_replay_keeps_places(tmp_path):
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": [7, 8, 9], "want": [2, 0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [5], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": [4], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "c", "tokens": [1, 2], "want": [1]}], "end": ["c", "b"]}]
    said, fake = [], FakeSession()
    trace.replay(fake, io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"), str(tmp_path), 2, said.append)
    assert said == [f"done {i}" for i in range(4)]
    assert fake.calls == [(0, 0, 3), (1, 0, 1), (0, 3, 1), (0, 0, 2)]
    assert np.fromfile(tmp_path / "0.f32", "<f4").tolist() == [0, 2, 9, 0, 0, 7]
    assert not (tmp_path / "1.f32").exists()
    assert np.fromfile(tmp_path / "2.f32", "<f4").tolist() == [0, 3, 4] and np.fromfile(tmp_path / "3.f32", "<f4").tolist() == [0, 1, 2]
