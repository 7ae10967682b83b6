"""Sugonex sessions on the GPU against the plain oracle (oracle/sugonex_oracle.py): every layer run's residual stream, logits of
whole prompts, portions and single tokens, batches, reused sequences, the edges of every window, generation, and the trace
runner.  float32 sessions are held to rounding; bf16 ones to a few bf16 roundings."""
import copy
import json
import os
import subprocess

import numpy as np
import pytest

import emel_cpp_b200 as eb
from emel_cpp_b200 import layered as ly
from emel_cpp_b200 import llama as el
from emel_cpp_b200 import models
from oracle import sugonex_oracle as so
from tests import sugonex_models as sm

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
# float32, bf16: rms of a row's error over the spread of the rows, worst row and mean
TOL = {True: 2e-5, False: 6e-2}
MEAN_TOL = {True: 5e-6, False: 1.5e-2}
LENGTHS = {"heads": 150, "odd": 83, "plain": 41, "tiled": 210}
BOTH = pytest.mark.parametrize("f32", [True, False], ids=["f32", "bf16"])
ALL = pytest.mark.parametrize("name", sorted(sm.MODELS))


@pytest.fixture(scope="module")
def be():
    b = eb.Backend(0)
    yield b
    b.close()


class Case:
    def __init__(self, cfg, folder, n, seed, change=None):
        self.cfg, self.folder = cfg, folder
        self.tensors = sm.tensors(cfg, seed)
        if change:
            change(self.tensors)
        sm.write_folder(folder, cfg, self.tensors)
        self.w = sm.as_f64(self.tensors)
        self.tokens = sm.random_tokens(cfg, n, seed + 1)
        self.streams = so.residual_streams(cfg, self.w, self.tokens)
        self.logits = so.head(cfg, self.w, self.streams[-1])

    def session(self, be, f32, n_ctx=256):
        return models.load(be, str(self.folder), n_ctx=n_ctx, float32=f32)


@pytest.fixture(scope="module")
def cases(tmp_path_factory):
    d = tmp_path_factory.mktemp("sugonex")
    return {name: Case(cfg, d / name, LENGTHS[name], 61) for name, cfg in sm.MODELS.items()}


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
def test_residual_stream_of_every_layer_run(be, cases, name, f32):
    c = cases[name]
    s = c.session(be, f32)
    n, W = len(c.tokens), c.cfg["width"]
    assert s.n_runs == len(c.streams)
    t = s.trace_layers(n)
    assert s.prefill(c.tokens, 0)
    got = t.reshape(-1)[:s.n_runs * n * W].reshape(s.n_runs, n, W)
    for l in range(s.n_runs):
        assert_close(sm.row_errors(got[l], c.streams[l]), f32, l)
    s.close()


@ALL
@BOTH
@pytest.mark.parametrize("sizes", [[4096], [1], [2], [3, 5, 2, 17], [64, 1, 7], [33], [63, 66]], ids=str)
def test_portions(be, cases, name, f32, sizes):
    c = cases[name]
    s = c.session(be, f32)
    assert_close(sm.row_errors(feed(s, c.tokens, sizes), c.logits), f32)
    s.close()


MECHANISMS = {
    "delta": sm.delta(2, 2, 32, 32, 1),
    "delta_conv": sm.delta(2, 2, 32, 32, 4),
    "delta_shared_heads": sm.delta(6, 2, 16, 64, 2),
    "latent": sm.windowed(4, 32, 32, 64, 0.4, 1000),
    "rotated_and_gated": sm.latent(4, 32, 32, 32, 64, 0.3, base=100.0),
    "window": sm.windowed(4, 32, 32, 64, 0.4, 7),
    "feed_forward": sm.windowed(2, 8, 8, 8, 1.0, 1, ff=96),
}


@BOTH
@pytest.mark.parametrize("what", sorted(MECHANISMS))
@pytest.mark.parametrize("around", ["alone", "loop", "cap"])
def test_each_mechanism_alone(be, tmp_path, what, around, f32):
    cfg = sm.model(48, 40, [MECHANISMS[what]], loop=(0, 1, 3) if around == "loop" else None, cap=2.0 if around == "cap" else None,
                   scale=1.0 if around == "alone" else 3.0)
    c = Case(cfg, tmp_path / "m", 70, 7)
    s = c.session(be, f32)
    for sizes in ([70], [1], [2, 9]):
        assert_close(sm.row_errors(feed(s, c.tokens, sizes), c.logits), f32, sizes)
    s.close()


@BOTH
@pytest.mark.parametrize("window", [1, 2, 17, 63, 64, 65, 100])
def test_window_edges(be, tmp_path, f32, window):
    """Scores so peaked that one key more or less is far above the tolerance."""
    cfg = sm.model(64, 50, [sm.windowed(4, 64, 64, 96, 0.7, window), sm.windowed(2, 32, 32, 48, 0.8, window, ff=32)])
    c = Case(cfg, tmp_path / "m", 140, 9)
    moved = []
    for by in (1, -1):
        if window + by < 1:
            continue
        bad = copy.deepcopy(cfg)
        for layer in bad["layers"]:
            layer["mixer"]["mask"]["size"] += by
        moved.append(sm.row_errors(so.logits(bad, c.w, c.tokens), c.logits).max())
    s = c.session(be, f32)
    for sizes in ([140], [1], [50, 3], [139, 1], [16, 64]):
        e = sm.row_errors(feed(s, c.tokens, sizes), c.logits)
        assert e.max() < 2 * TOL[f32], (sizes, int(e.argmax()), e.max())
        assert min(moved) > 2.5 * e.max(), (moved, e.max())
    s.close()


@BOTH
@pytest.mark.parametrize("rot", [0, 32])
def test_far_key_found_by_one_query(be, tmp_path, f32, rot):
    """One token's query meets one token's key (equal directions, scaled up): a key 290 tokens back decides the logits."""
    kind = sm.latent(2, 64, rot, 64, 64, 0.125, base=1e6) if rot else sm.windowed(2, 64, 64, 64, 0.125, 400)
    cfg = sm.model(64, 40, [kind])

    def point(t):
        # the latent direction of token 3 through every head's key rows becomes the query of token 7
        n3 = t["embed"][3] / np.sqrt(np.mean(t["embed"][3] ** 2)) * (1 + t["l0.norm1"])
        n7 = t["embed"][7] / np.sqrt(np.mean(t["embed"][7] ** 2)) * (1 + t["l0.norm1"])
        lat = t["l0.mix.dkv"][:64] @ n3
        lat = lat / np.sqrt(np.mean(lat ** 2)) * t["l0.mix.dkv.norm"]
        for h in range(2):
            key = t["l0.mix.uk"][64 * h:64 * h + 64] @ lat
            at = (64 + rot) * h
            t["l0.mix.q"][at:at + 64] = sm.round_bf16(t["l0.mix.q"][at:at + 64] + 0.02 * np.outer(key, n7))
    c = Case(cfg, tmp_path / "m", 1, 77, change=point)
    toks = [t if t not in (3, 7) else 0 for t in sm.random_tokens(cfg, 300, 5)]
    toks[9], toks[299] = 3, 7
    want = so.logits(cfg, c.w, toks)
    other = list(toks)
    other[9] = 0
    assert sm.row_errors(so.logits(cfg, c.w, other), want)[299] > 0.3
    s = models.load(be, str(c.folder), n_ctx=300, float32=f32)
    for sizes in ([300], [299, 1], [150, 149, 1], [298, 2], [1]):
        assert sm.row_errors(feed(s, toks, sizes), want)[[100, 298, 299]].max() < TOL[f32], sizes
    s.close()


@BOTH
def test_state_remembers_a_far_token(be, tmp_path, f32):
    """A delta layer that hardly forgets: what one early token wrote is read hundreds of tokens later."""
    cfg = sm.model(64, 40, [sm.delta(2, 1, 64, 64, 2)])

    def keep(t):
        t["l0.mix.A_log"] = np.full(2, -10.0, np.float32)
        # only token 3 writes: beta follows its direction, and is near zero for the others
        n3 = t["embed"][3] / np.linalg.norm(t["embed"][3])
        t["embed"] -= np.outer(t["embed"] @ n3 + 4.0, n3)
        t["embed"][3] = 8.0 * n3
        t["embed"] = sm.round_bf16(t["embed"])
        t["l0.mix.b"] = sm.round_bf16(np.stack([n3, n3]) * 2.0)
    c = Case(cfg, tmp_path / "m", 1, 78, change=keep)
    toks = [t if t != 3 else 0 for t in sm.random_tokens(cfg, 400, 5)]
    toks[5] = 3
    want = so.logits(cfg, c.w, toks)
    other = list(toks)
    other[5] = 0
    assert sm.row_errors(so.logits(cfg, c.w, other), want)[399] > 0.1
    s = models.load(be, str(c.folder), n_ctx=400, float32=f32)
    for sizes in ([400], [1], [64, 335, 1], [6, 2, 50]):
        assert_close(sm.row_errors(feed(s, toks, sizes), want), f32, sizes)
    s.close()


@BOTH
def test_repeated_keys(be, tmp_path, f32):
    """Long runs of the same few tokens with step sizes near 1 and hardly any decay: within a chunk every key meets itself
    many times, so that the triangular systems of the chunked recurrence are far from the identity."""
    cfg = sm.model(64, 30, [sm.delta(3, 1, 32, 40, 1), sm.delta(2, 2, 64, 32, 2)], loop=(0, 2, 2))

    def near_one(t):
        for i in (0, 1):
            t[f"l{i}.mix.A_log"] = np.full_like(t[f"l{i}.mix.A_log"], -9.0)
            t[f"l{i}.mix.b"] = sm.round_bf16(4.0 * t[f"l{i}.mix.b"])
    c = Case(cfg, tmp_path / "m", 1, 12, change=near_one)
    toks = [5] * 40 + [7, 5] * 40 + [9] * 70 + [5, 5, 7, 9] * 10
    want = so.logits(cfg, c.w, toks)
    s = models.load(be, str(c.folder), n_ctx=240, float32=f32)
    for sizes in ([300], [1], [64, 3, 61]):
        assert_close(sm.row_errors(feed(s, toks, sizes), want), f32, sizes)
    s.close()


@BOTH
def test_first_tokens(be, cases, f32):
    c = cases["odd"]
    s = c.session(be, f32)
    for n in (1, 2, 3, 4, 5):
        assert sm.row_errors(feed(s, c.tokens[:n], [n]), c.logits[:n]).max() < TOL[f32]
        assert sm.row_errors(feed(s, c.tokens[:n + 1], [n, 1]), c.logits[:n + 1]).max() < TOL[f32]
    s.close()


@BOTH
def test_long_decoding(be, cases, f32):
    c = cases["tiled"]
    s = c.session(be, f32)
    n0 = 11
    assert s.prefill(c.tokens[:n0], 0)
    got = np.stack([s.decode(t, n0 + i, want_logits=True) for i, t in enumerate(c.tokens[n0:])])
    assert_close(sm.row_errors(got, c.logits[n0:]), f32)
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
            e = sm.row_errors(logits[j:j + 1], c.logits[n - 1 + step:n + step])
            assert e.max() < TOL[f32], (step, j, e.max())
            assert ids[j] == int(np.argmax(logits[j]))
    s.close()


@BOTH
@pytest.mark.parametrize("name", ["odd", "tiled"])
def test_sequences_used_again(be, cases, name, f32):
    """A sequence that starts at position 0 forgets what its slot held; other sequences keep theirs."""
    c = cases[name]
    s = c.session(be, f32)
    assert s.set_sequences(3)
    other = sm.random_tokens(c.cfg, 70, 99)
    assert s.select_sequence(1) and s.prefill(c.tokens[:20], 0)
    for again in range(2):
        for slot in (0, 2):
            assert s.select_sequence(slot)
            assert s.prefill(other[:60 - 13 * again], 0)
            for i in range(3):
                s.decode(other[i], 60 - 13 * again + i)
            for sizes in ([2], [300], [1]):
                assert_close(sm.row_errors(feed(s, c.tokens, sizes), c.logits), f32, again, slot, sizes)
    assert s.select_sequence(1)
    assert sm.row_errors(feed(s, c.tokens[20:], [7], start=20), c.logits[20:]).max() < TOL[f32]
    s.close()


@ALL
def test_greedy_generation(be, cases, name):
    c = cases[name]
    s = c.session(be, True)
    prompt, n = c.tokens[:15], 12
    want, toks = [], list(prompt)
    for _ in range(n):
        row = so.logits(c.cfg, c.w, toks)[-1]
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


@BOTH
def test_prompt_in_small_batches(be, cases, f32):
    c = cases["tiled"]
    s = c.session(be, f32)
    assert s.set_prefill_batch(48)
    assert_close(sm.row_errors(feed(s, c.tokens, [500]), c.logits), f32)
    assert s.set_prefill_batch(0)
    assert_close(sm.row_errors(feed(s, c.tokens, [500]), c.logits), f32)
    s.close()


@BOTH
def test_long_prompts(be, tmp_path, f32):
    """Prompts of many chunks of the delta rule and many key tiles, whole, cut and continued."""
    cfg = sm.model(96, 60, [sm.delta(4, 2, 32, 64, 4, ff=64), sm.latent(4, 32, 16, 32, 40, 0.4, base=5000.0, ff=48),
                            sm.windowed(3, 48, 64, 56, 0.4, 330, ff=32), sm.delta(2, 2, 64, 32, 3)], loop=(0, 2, 2))
    c = Case(cfg, tmp_path / "m", 1150, 41)
    s = c.session(be, f32, n_ctx=1152)
    for sizes in ([1150], [700, 449, 1], [1, 600, 549], [511, 3, 636], [1088, 1]):
        assert_close(sm.row_errors(feed(s, c.tokens, sizes), c.logits), f32, sizes)
    s.close()


def test_post_norm_stack_with_the_same_mixers(be):
    """The mixers are not tied to the parallel arrangement: post-norm sublayers around a delta and a latent layer, looped,
    with RMS norms, biases and silu."""
    g = np.random.default_rng(3)
    W, V, ff, n = 64, 50, 72, 45
    layers = [ly.delta_layer(4, 2, 16, 24, 3, n_ff=ff, ff_act=ly.FF_SILU, ff_bias=True),
              ly.latent_layer(3, 20, 28, 33, 0.4, rope_dim=8, rope_freq_base=300.0, out_gate=True)]
    s = ly.Session(be, ly.config(2, W, V, 64, 1e-5), layers, True, ly.stack(ly.STACK_POST_NORM, ly.NORM_RMS, loop=(0, 2, 2), loop_step=True))

    def mat(layer, role, *shape):
        a = sm.round_bf16(g.standard_normal(shape) * 1.2 / np.sqrt(shape[1]))
        assert s.load_matrix(layer, role, sm_bits(a)), role
        return a.astype(np.float64)

    def vec(layer, role, *shape, base=1.0):
        a = sm.round_bf16(base + 0.3 * g.standard_normal(shape))
        assert s.load_vector(layer, role, a), role
        return a.astype(np.float64)

    from emel_cpp_b200 import safetensors as st
    sm_bits = st.f32_to_bf16
    embed, head, final, step = mat(-1, el.TOKEN_EMBD, V, W), mat(-1, el.OUTPUT, V, W), vec(-1, el.OUTPUT_NORM, W), vec(-1, ly.LOOP_STEP, 2, W, base=0.0)
    w = {}
    rows = mat(0, ly.MIX_IN, ly.in_rows(layers[0]), W)
    at = 0
    for name, k in (("q", 32), ("k", 32), ("v", 96), ("g", 96), ("b", 4), ("a", 4)):
        w["0." + name] = rows[at:at + k]
        at += k
    conv = vec(0, ly.MIX_CONV, 160, 3, base=0.4)
    w["0.q.conv"], w["0.k.conv"], w["0.v.conv"] = conv[:32], conv[32:64], conv[64:]
    w["0.A_log"], w["0.dt_bias"], w["0.norm"] = vec(0, ly.MIX_DECAY_LOG, 4, base=-1.0), vec(0, ly.MIX_STEP_BIAS, 4, base=0.0), vec(0, ly.MIX_NORM_OUT, 24)
    rows = mat(1, ly.MIX_IN, ly.in_rows(layers[1]), W)
    w["1.q"], w["1.g"], w["1.dkv"] = rows[:84], rows[84:168], rows[168:]
    w["1.dkv.norm"] = vec(1, ly.MIX_LATENT_NORM, 33)
    up = mat(1, ly.MIX_LATENT_UP, 3 * 48, 33)
    w["1.uk"], w["1.uv"] = up[:60], up[60:]
    w["0.o"], w["1.o"] = mat(0, el.ATTN_OUT, W, 96), mat(1, el.ATTN_OUT, W, 84)
    norms = [vec(0, el.ATTN_NORM, W), vec(1, el.ATTN_NORM, W)]
    fin, fib, fd, fdb = mat(0, ly.FFN_IN, 2 * ff, W), vec(0, ly.FFN_IN_BIAS, 2 * ff, base=0.0), mat(0, el.FFN_DOWN, W, ff), vec(0, ly.FFN_DOWN_BIAS, W, base=0.0)
    norm_ff = vec(0, el.FFN_NORM, W)
    toks = g.integers(0, V, n).tolist()
    x = embed[toks]
    for t in range(2):
        x = x + step[t]
        y = so.delta_mixer(x, w, "0.", {"heads": 4, "kv_heads": 2, "dim": 16, "vdim": 24}, 1e-5)
        x = x + so.rms_norm(y, norms[0], 1e-5)
        gu = x @ fin.T + fib
        x = x + so.rms_norm((so.silu(gu[:, :ff]) * gu[:, ff:]) @ fd.T + fdb, norm_ff, 1e-5)
        y = so.latent_mixer(x, w, "1.", {"heads": 3, "dim": 20, "rot_dim": 8, "vdim": 28, "kv_rank": 33, "scale": 0.4, "rot": {"base": 300.0}}, 1e-5, True)
        x = x + so.rms_norm(y, norms[1], 1e-5)
    want = so.rms_norm(x, final, 1e-5) @ head.T
    for sizes in ([n], [1], [7, 2, 20]):
        assert_close(sm.row_errors(feed(s, toks, sizes), want), True, sizes)
    s.close()


def test_requests_are_checked(be, cases):
    c = cases["odd"]
    s = c.session(be, False, n_ctx=32)
    assert s.prefill(c.tokens[:5], 0)
    assert not s.prefill(c.tokens[:2], 3) and s.last_error == eb.INVALID_REQUEST     # back
    assert not s.prefill(c.tokens[:2], 7)                                            # ahead
    assert not s.prefill(c.tokens[:28], 5)                                           # past the context
    s.decode(1, 5)
    s.decode(1, 0)                                                                   # starts again
    assert not s.load_matrix(1, el.ATTN_OUT, np.zeros((c.cfg["width"], 168), np.uint16))   # set beside the down projection instead
    assert not s.load_vector(1, ly.MIX_LATENT_NORM, np.zeros(3, np.float32))               # a delta layer has none
    assert not s.load_vector(1, ly.FFN_IN_BIAS, np.zeros(100, np.float32))                 # no biases in this design
    s.close()


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
        assert sm.row_errors(got, c.logits[rows]).max() < 1.5 * TOL[f32], step
    assert not (tmp_path / "1.f32").exists()
