"""Metulix sessions on the GPU against the plain oracle (oracle/metulix_oracle.py): every layer's residual stream,
logits of whole prompts, portions and single tokens, batches, reused sequences, the edges of every mask, generation,
and the trace runner.  float32 sessions are held to rounding; bf16 ones to a few bf16 roundings."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import emel_cpp_b200 as eb
from emel_cpp_b200 import layered as ly
from emel_cpp_b200 import llama as el
from emel_cpp_b200 import models
from oracle import metulix_oracle as mo
from tests import metulix_models as mm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# float32, bf16: rms of a row's error over the spread of the rows.  (A bf16 row whose sublayer output nearly cancels before
# its norm may be several times worse than the others, hence the looser bound on single rows beside the one on the mean.)
TOL = {True: 2e-5, False: 0.12}
MEAN_TOL = {True: 4e-6, False: 1.2e-2}
LENGTHS = {"heads": 150, "odd": 83, "plain": 41, "tiled": 210}
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])
ALL = pytest.mark.parametrize("name", sorted(mm.MODELS))


@pytest.fixture(scope="module")
def be():
    b = eb.Backend(0)
    yield b
    b.close()


class Case:
    def __init__(self, cfg, folder, n, seed):
        self.cfg, self.folder = cfg, folder
        self.tensors = mm.tensors(cfg, seed)
        mm.write_folder(folder, cfg, self.tensors)
        self.w = mm.as_f64(self.tensors)
        self.tokens = mm.random_tokens(cfg, n, seed + 1)
        self.streams = mo.residual_streams(cfg, self.w, self.tokens)
        self.logits = mo.logits(cfg, self.w, self.tokens)

    def session(self, be, f32, n_ctx=256):
        return models.load(be, str(self.folder), n_ctx=n_ctx, float32=f32)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    d = tmp_path_factory.mktemp("metulix")
    return {name: Case(cfg, d / name, LENGTHS[name], 31) for name, cfg in mm.MODELS.items()}


def assert_close(e, f32, *where):
    assert e.max() < TOL[f32] and e.mean() < MEAN_TOL[f32], (*where, int(e.argmax()), float(e.max()), float(e.mean()))


def feed(sess, tokens, sizes, start=0):
    """Logits of every position, the tokens cut into portions of the given sizes (the last one repeats)."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(i, len(sizes) - 1)], len(tokens) - at)
        out.append(sess.prefill_logits(tokens[at:at + n], start + at, range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)


@ALL
@BOTH
def test_residual_stream_of_every_layer(be, cases, name, f32):
    c = cases[name]
    s = c.session(be, f32)
    n, L, W = len(c.tokens), len(c.cfg["layers"]), c.cfg["width"]
    t = s.trace_layers(n)
    assert s.prefill(c.tokens, 0)
    got = t.reshape(-1)[:L * n * W].reshape(L, n, W)
    for l in range(L):
        e = mm.row_errors(got[l], c.streams[l])
        assert_close(e, f32, l)
    s.close()


@ALL
@BOTH
@pytest.mark.parametrize("sizes", [[4096], [1], [2], [3, 5, 2, 17], [64, 1, 7], [33]], ids=str)
def test_portions(be, cases, name, f32, sizes):
    c = cases[name]
    s = c.session(be, f32)
    e = mm.row_errors(feed(s, c.tokens, sizes), c.logits)
    assert_close(e, f32)
    s.close()


def single_layer(kind, **changes):
    """One layer with one mechanism, the others off."""
    d = dict(n_head=4, n_head_kv=2, key_dim=24, value_dim=32, scale=0.4, norm_qk=False, norm_v=False, mix_heads=False)
    d.update(changes)
    if kind == "linear":
        return ly.linear_layer(3, d["key_dim"], d["value_dim"], [0.6, 0.99, 0.9])
    return ly.attention_layer(**d)


@BOTH
@pytest.mark.parametrize("what", ["plain", "conv", "norm_qk", "norm_v", "rope", "mix", "window", "keep", "linear", "ff"])
def test_each_mechanism_alone(be, what, f32):
    g = np.random.default_rng(len(what))
    W, V, n = 48, 40, 50
    ch = {"conv": dict(conv_taps=4), "norm_qk": dict(norm_qk=True), "norm_v": dict(norm_v=True), "rope": dict(rope_dim=16, rope_freq_base=100.0),
          "mix": dict(mix_heads=True), "window": dict(window=7), "keep": dict(window=6, keep_first=4), "ff": dict(n_ff=72)}.get(what, {})
    l = single_layer("linear" if what == "linear" else "attention", **ch)
    heads, kv = l.n_head, l.n_head_kv
    s = ly.Session(be, ly.config(1, W, V, 64, 1e-5), [l], f32)

    def mat(layer, role, rows, k):
        a = mm.round_bf16(g.standard_normal((rows, k)) * 1.3 / np.sqrt(k))
        assert s.load_matrix(layer, role, mm.st.f32_to_bf16(a)), role
        return a.astype(np.float64)

    def vec(layer, role, *shape):
        a = mm.round_bf16(0.8 + 0.4 * g.standard_normal(shape))
        assert s.load_vector(layer, role, a), role
        return a.astype(np.float64)

    embed, head = mat(-1, el.TOKEN_EMBD, V, W), mat(-1, el.OUTPUT, V, W)
    w = {"embed": embed, "head": head, "final.norm": vec(-1, el.OUTPUT_NORM, W), "l0.norm1": vec(0, el.ATTN_NORM, W)}
    stacked = mat(0, ly.MIX_IN, ly.in_rows(l), W)
    hd, hv = heads * l.key_dim, heads * l.value_dim
    if what == "linear":
        cuts = dict(q=hd, k=hd, v=hv, g=hv)
        w["l0.mix.norm"] = vec(0, ly.MIX_NORM_OUT, hv)
        cfg_l = mm.lightning(heads, l.key_dim, l.value_dim, [l.decay[i] for i in range(heads)])
    else:
        cuts = dict(q=hd, k=kv * l.key_dim, v=kv * l.value_dim)
        cfg_l = mm.attention(heads, kv, l.key_dim, l.value_dim, 0.4, conv=l.conv_taps, rot=(l.rope_dim, l.rope_freq_base),
                             window=l.window or None, keep=l.keep_first, ff=l.n_ff or None)
        cfg_l["mixer"]["norm_v"] = bool(l.norm_v)
    conv = vec(0, ly.MIX_CONV, len(stacked), l.conv_taps) if l.conv_taps else None
    at = 0
    for n_, rows in cuts.items():
        w["l0.mix." + n_] = stacked[at:at + rows]
        if conv is not None:
            w[f"l0.mix.{n_}.conv"] = conv[at:at + rows]
        at += rows
    if l.norm_qk:
        w["l0.mix.q.norm"], w["l0.mix.k.norm"] = vec(0, ly.MIX_NORM_Q, hd), vec(0, ly.MIX_NORM_K, kv * l.key_dim)
    if l.mix_heads:
        w["l0.mix.talk"] = vec(0, ly.MIX_HEADS, heads, heads)
    w["l0.mix.o"] = mat(0, el.ATTN_OUT, W, hv)
    if l.n_ff:
        ff_in = mat(0, ly.FFN_IN, 2 * l.n_ff, W)
        b = vec(0, ly.FFN_IN_BIAS, 2 * l.n_ff)
        w.update({"l0.norm2": vec(0, el.FFN_NORM, W), "l0.mlp.gate": ff_in[:l.n_ff], "l0.mlp.up": ff_in[l.n_ff:],
                  "l0.mlp.gate.b": b[:l.n_ff], "l0.mlp.up.b": b[l.n_ff:], "l0.mlp.down": mat(0, el.FFN_DOWN, W, l.n_ff),
                  "l0.mlp.down.b": vec(0, ly.FFN_DOWN_BIAS, W)})
    cfg = mm.model(W, V, [cfg_l], eps=1e-5)
    toks = mm.random_tokens(cfg, n, 3)
    want = mo.logits(cfg, w, toks)
    for sizes in ([64], [1], [2, 9]):
        e = mm.row_errors(feed(s, toks, sizes), want)
        assert_close(e, f32, sizes)
    s.close()


def standing_out(cfg, window, keep, f):
    """`cfg` with the mask changed by f and its scale raised, so that single keys carry the weights."""
    c = copy.deepcopy(cfg)
    for layer in c["layers"]:
        m = layer["mixer"]
        if layer["type"] == "attention":
            m["scale"] *= 4.0
            m["mask"] = {"size": window, "keep_first": keep}
    f(c)
    return c


@BOTH
@pytest.mark.parametrize("window,keep", [(64, 3), (65, 1), (17, 16), (100, 0), (1, 2)])
def test_mask_edges(be, tmp_path, f32, window, keep):
    """Scores so peaked that one key more or less at either edge of the mask is far above the tolerance."""
    base = mm.model(64, 50, [mm.attention(4, 2, 64, 64, 0.3, conv=2, rot=(32, 1000.0), ff=96), mm.lightning(1, 32, 32, [0.9]),
                             mm.attention(4, 2, 64, 64, 0.3, conv=2, rot=(32, 1000.0), kv_from=0)])
    cfg = standing_out(base, window, keep, lambda c: None)
    c = Case(cfg, tmp_path / "m", 140, 9)
    moved = []
    for key, by in (("size", 1), ("size", -1), ("keep_first", 1), ("keep_first", -1)):
        if cfg["layers"][0]["mixer"]["mask"][key] + by < (1 if key == "size" else 0):
            continue

        def change(cc, key=key, by=by):
            for layer in cc["layers"]:
                if layer["type"] == "attention":
                    layer["mixer"]["mask"][key] += by
        bad = mo.logits(standing_out(base, window, keep, change), c.w, c.tokens)
        moved.append(mm.row_errors(bad, c.logits).max())
    s = c.session(be, f32)
    tol = 2 * TOL[f32]
    for sizes in ([140], [1], [50, 3]):
        e = mm.row_errors(feed(s, c.tokens, sizes), c.logits)
        assert e.max() < tol, (sizes, int(e.argmax()), e.max())
        assert min(moved) > 2.5 * e.max(), (moved, e.max())
    s.close()


@BOTH
def test_far_key_found_by_one_query(be, tmp_path, f32):
    """One token's query meets one token's key (equal directions, scaled up): the kept token of a long prompt, far
    outside the window, decides the logits; with it hidden they are elsewhere."""
    cfg = mm.model(64, 40, [mm.attention(2, 1, 64, 64, 0.125, conv=1, rot=(0, 1.0), window=20, keep=4)])
    t = mm.tensors(cfg, 77)
    # without rotation or taps, token 7's query and token 3's key both follow direction e: their product is large
    t["l0.mix.q.conv"], t["l0.mix.k.conv"] = np.ones_like(t["l0.mix.q.conv"]), np.ones_like(t["l0.mix.k.conv"])
    for n in ("q", "k"):
        t[f"l0.mix.{n}.norm"] = mm.round_bf16(3.0 * t[f"l0.mix.{n}.norm"])
    e = t["l0.mix.k"] @ t["embed"][3]
    for h in range(2):
        t["l0.mix.q"][64 * h:64 * h + 64] = mm.round_bf16(t["l0.mix.q"][64 * h:64 * h + 64] + np.outer(e, t["embed"][7]) / 30)
    folder = mm.write_folder(tmp_path / "m", cfg, t)
    toks = [t_ if t_ not in (3, 7) else 0 for t_ in mm.random_tokens(cfg, 300, 5)]
    toks[2], toks[299] = 3, 7
    w = mm.as_f64(t)
    want = mo.logits(cfg, w, toks)
    hidden = copy.deepcopy(cfg)
    hidden["layers"][0]["mixer"]["mask"]["keep_first"] = 2
    assert mm.row_errors(mo.logits(hidden, w, toks), want)[299] > 0.3
    s = models.load(be, folder, n_ctx=300, float32=f32)
    for sizes in ([300], [299, 1], [150, 149, 1]):
        assert mm.row_errors(feed(s, toks, sizes), want)[[100, 298, 299]].max() < TOL[f32]
    s.close()


@BOTH
def test_first_tokens(be, cases, f32):
    c = cases["odd"]
    s = c.session(be, f32)
    for n in (1, 2, 3, 4, 5):
        assert mm.row_errors(feed(s, c.tokens[:n], [n]), c.logits[:n]).max() < TOL[f32]
        assert mm.row_errors(feed(s, c.tokens[:n + 1], [n, 1]), c.logits[:n + 1]).max() < TOL[f32]
    s.close()


@BOTH
def test_long_decoding(be, cases, f32):
    c = cases["tiled"]
    s = c.session(be, f32)
    n0 = 11
    assert s.prefill(c.tokens[:n0], 0)
    got = np.stack([s.decode(t, n0 + i, want_logits=True) for i, t in enumerate(c.tokens[n0:])])
    e = mm.row_errors(got, c.logits[n0:])
    assert_close(e, f32)
    s.close()


@ALL
@BOTH
def test_batches_of_unequal_sequences(be, cases, name, f32):
    """Sequences with prompts of different lengths stepped together, each against itself alone."""
    c = cases[name]
    s = c.session(be, f32)
    lens = [1, 9, 30, 2, 40]
    assert s.set_sequences(len(lens))
    for j, n in enumerate(lens):
        assert s.select_sequence(j)
        if n > 1:
            assert s.prefill(c.tokens[:n - 1], 0)
    for step in range(6):
        if max(lens) + step > len(c.tokens):
            break
        toks = [c.tokens[n - 1 + step] for n in lens]
        ids, logits = s.decode_batch(toks, [n - 1 + step for n in lens], want_logits=True)
        for j, n in enumerate(lens):
            e = mm.row_errors(logits[j:j + 1], c.logits[n - 1 + step:n + step])
            assert e.max() < TOL[f32], (step, j, e.max())
            assert ids[j] == int(np.argmax(logits[j]))
    s.close()


@BOTH
def test_sequences_used_again(be, cases, f32):
    """A sequence that starts at position 0 forgets what its slot held; other sequences keep theirs."""
    c = cases["odd"]
    s = c.session(be, f32)
    assert s.set_sequences(3)
    other = mm.random_tokens(c.cfg, 70, 99)
    assert s.select_sequence(1) and s.prefill(c.tokens[:20], 0)
    for again in range(3):
        for slot in (0, 2):
            assert s.select_sequence(slot)
            assert s.prefill(other[:70 - 13 * again], 0)
            for i in range(3):
                s.decode(other[i], 70 - 13 * again + i)
            for sizes in ([2], [83], [1]):
                e = mm.row_errors(feed(s, c.tokens, sizes), c.logits)
                assert_close(e, f32, again, slot, sizes)
    assert s.select_sequence(1)
    assert mm.row_errors(feed(s, c.tokens[20:], [7], start=20), c.logits[20:]).max() < TOL[f32]
    s.close()


@ALL
def test_greedy_generation(be, cases, name):
    c = cases[name]
    s = c.session(be, True)
    prompt, n = c.tokens[:15], 12
    want, toks = [], list(prompt)
    for _ in range(n):
        row = mo.logits(c.cfg, c.w, toks)[-1]
        top = np.sort(row)[-2:]
        want.append(int(np.argmax(row)))
        assert top[1] - top[0] > 1e-4      # no near tie the rounding could turn
        toks.append(want[-1])
    assert s.prefill(prompt[:-1], 0)
    assert list(s.generate(prompt[-1], len(prompt) - 1, n)) == want
    # again through the batch loop, in two sequences that are at different places
    assert s.set_sequences(2)
    for j, cut in ((0, 15), (1, 6)):
        assert s.select_sequence(j) and s.prefill(toks[:cut - 1], 0)
    ids = s.generate_batch([toks[14], toks[5]], [14, 5], 8)
    assert list(ids[:, 0]) == want[:8]
    assert s.launches_per_token() > 0
    # one sequence goes on where the batch left it
    assert s.select_sequence(0)
    assert list(s.generate(want[7], 15 + 7, 3)) == want[8:11]
    s.close()


def test_prompt_in_small_batches(be, cases):
    c = cases["tiled"]
    s = c.session(be, True)
    assert s.set_prefill_batch(48)
    assert mm.row_errors(feed(s, c.tokens, [500]), c.logits).max() < TOL[True]
    assert s.set_prefill_batch(0)
    assert mm.row_errors(feed(s, c.tokens, [500]), c.logits).max() < TOL[True]
    s.close()


def test_requests_are_checked(be, cases):
    c = cases["odd"]
    s = c.session(be, False, n_ctx=32)
    assert s.prefill(c.tokens[:5], 0)
    assert not s.prefill(c.tokens[:2], 3) and s.last_error == eb.INVALID_REQUEST     # back
    assert not s.prefill(c.tokens[:2], 7)                                            # ahead
    assert not s.prefill(c.tokens[:28], 5)                                           # past the context
    assert not s.prefill([c.cfg["vocab"]], 5)
    for bad in ([1, 0], [0, 0], [3], [-1]):
        with pytest.raises(eb.BackendError):
            s.prefill_logits(c.tokens[:3], 5, bad)
    with pytest.raises(eb.BackendError):
        s.decode(1, 4)
    s.decode(1, 5)
    s.decode(1, 0)                                                                   # starts again
    assert not s.set_window(None) or s.last_error in (eb.OK, eb.UNSUPPORTED_OP)
    assert not s.load_vector(0, ly.MIX_CONV, np.zeros(3, np.float32))           # a linear layer has none
    assert not s.load_matrix(1, ly.MIX_IN, np.zeros((5, 5), np.uint16))
    s.close()


def test_llama_prompt_logits(be, port):
    """prefill_logits of a block-quantized session: the rows decode() gives for the same prefix."""
    from tests.test_gpu_decoder import TINY, build_model
    sess, cpu = build_model(be, port, TINY, {"embd": eb.Q4_K, "output": eb.Q6_K, "default": eb.Q4_K}, seed=13)
    cpu.close()
    toks = np.random.default_rng(1).integers(0, TINY["n_vocab"], 40).tolist()
    got = sess.prefill_logits(toks, 0, [0, 7, 39])
    for row, i in zip(got, (0, 7, 39)):
        if i:
            assert sess.prefill(toks[:i], 0)
        assert mm.row_errors(row[None], sess.decode(toks[i], i, want_logits=True)[None]).max() < 5e-2
    sess.close()


@BOTH
def test_trace_runner(cases, tmp_path, f32):
    c = cases["odd"]
    a, b = c.tokens, c.tokens[:31]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:40], "want": [39, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[40:41], "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b[2:], "want": list(range(29))}], "end": ["b"]},
             {"step": 4, "entries": [{"id": "c", "tokens": b, "want": [30]}], "end": ["c"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(c.folder), "--dtype", "float32" if f32 else "bfloat16",
                        "--out", str(tmp_path), "--max-tokens", "90"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, timeout=600, cwd=str(tmp_path))
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
    for step, rows in ((0, [39, 3]), (2, [40]), (3, list(range(2, 31))), (4, [30])):
        got = np.fromfile(tmp_path / f"{step}.f32", "<f4").reshape(len(rows), -1)
        assert mm.row_errors(got, c.logits[rows]).max() < 1.5 * TOL[f32], step
    assert not (tmp_path / "1.f32").exists()


@BOTH
def test_long_prompts(be, tmp_path, f32):
    """Prompts of several key strips and several segments of the linear state, whole, cut and continued."""
    cfg = mm.model(96, 60, [mm.lightning(2, 48, 40, [0.999, 0.97], ff=64), mm.attention(4, 2, 32, 32, 0.5, conv=3, rot=(32, 5000.0), window=330, keep=7),
                            mm.lightning(3, 32, 72, [0.9995, 0.6, 1.0]), mm.attention(4, 2, 32, 32, 0.5, conv=2, rot=(32, 5000.0), kv_from=1)])
    cfg["layers"][3]["mixer"].pop("mask", None)     # the borrowing layer sees everything
    c = Case(cfg, tmp_path / "m", 1150, 41)
    s = c.session(be, f32, n_ctx=1152)
    for sizes in ([1150], [700, 449, 1], [1, 600, 549], [511, 3, 636]):
        assert_close(mm.row_errors(feed(s, c.tokens, sizes), c.logits), f32, sizes)
    s.close()
