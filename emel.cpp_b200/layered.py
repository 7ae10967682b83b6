"""Layered decoder sessions (include/emelb_llama.h, emelb_llama_create_stack): a decoder described layer by layer,
stepped through the same session calls as the block-quantized one."""
from __future__ import annotations

import ctypes as C

import numpy as np

import emel_cpp_b200 as eb
from emel_cpp_b200 import llama as el

MIXER_ATTENTION, MIXER_LINEAR, MIXER_LATENT, MIXER_DELTA = range(4)
(MIX_IN, MIX_CONV, MIX_NORM_Q, MIX_NORM_K, MIX_HEADS, MIX_NORM_OUT, FFN_IN, FFN_IN_BIAS, FFN_DOWN_BIAS, MIX_LATENT_NORM, MIX_LATENT_UP,
 MIX_DECAY_LOG, MIX_STEP_BIAS, LAYER_OUT, LOOP_STEP) = range(12, 27)
FF_SILU, FF_GELU_TANH = 0, 1
STACK_POST_NORM, STACK_PARALLEL = 0, 1
NORM_LAYER, NORM_RMS = 0, 1


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class LayerConfig(C.Structure):
    _fields_ = [("mixer", C.c_int32), ("n_head", C.c_int32), ("n_head_kv", C.c_int32), ("key_dim", C.c_int32),
                ("value_dim", C.c_int32), ("conv_taps", C.c_int32), ("norm_qk", C.c_int32), ("norm_v", C.c_int32),
                ("mix_heads", C.c_int32), ("rope_dim", C.c_int32), ("rope_freq_base", C.c_float),
                ("attn_scale", C.c_float), ("window", C.c_int32), ("keep_first", C.c_int32), ("kv_from", C.c_int32),
                ("n_ff", C.c_int32), ("decay", C.POINTER(C.c_float)), ("rope_half", C.c_int32), ("kv_rank", C.c_int32),
                ("out_gate", C.c_int32), ("ff_act", C.c_int32), ("ff_bias", C.c_int32)]


class StackConfig(C.Structure):
    _fields_ = [("arrangement", C.c_int32), ("norm", C.c_int32), ("loop_start", C.c_int32), ("loop_stop", C.c_int32),
                ("loop_times", C.c_int32), ("loop_step", C.c_int32), ("logit_scale", C.c_float), ("logit_softcap", C.c_float)]


def stack(arrangement=STACK_POST_NORM, norm=NORM_LAYER, loop=None, loop_step=False, logit_scale=1.0, logit_softcap=0.0) -> StackConfig:
    """loop: (first layer, layer behind the last, passes)."""
    start, stop, times = loop or (0, 0, 0)
    return StackConfig(arrangement, norm, start, stop, times, int(loop_step), logit_scale, logit_softcap)


def linear_layer(n_head, key_dim, value_dim, decay, n_ff=0, ff_act=FF_SILU, ff_bias=True) -> LayerConfig:
    if len(decay) != n_head:
        raise ValueError(f"{len(decay)} decays for {n_head} heads")
    l = LayerConfig(mixer=MIXER_LINEAR, n_head=n_head, key_dim=key_dim, value_dim=value_dim, kv_from=-1, n_ff=n_ff, ff_act=ff_act,
                    ff_bias=int(ff_bias))
    l._decay = (C.c_float * n_head)(*[float(d) for d in decay])   # alive as long as the description
    l.decay = C.cast(l._decay, C.POINTER(C.c_float))
    return l


def attention_layer(n_head, n_head_kv, key_dim, value_dim, scale, conv_taps=0, norm_qk=True, norm_v=True, mix_heads=True,
                    rope_dim=0, rope_freq_base=10000.0, window=0, keep_first=0, kv_from=-1, n_ff=0, ff_act=FF_SILU, ff_bias=True) -> LayerConfig:
    return LayerConfig(mixer=MIXER_ATTENTION, n_head=n_head, n_head_kv=n_head_kv, key_dim=key_dim, value_dim=value_dim,
                       conv_taps=conv_taps, norm_qk=int(norm_qk), norm_v=int(norm_v), mix_heads=int(mix_heads),
                       rope_dim=rope_dim, rope_freq_base=rope_freq_base, attn_scale=scale, window=window,
                       keep_first=keep_first, kv_from=kv_from, n_ff=n_ff, ff_act=ff_act, ff_bias=int(ff_bias))


def latent_layer(n_head, key_dim, value_dim, kv_rank, scale, rope_dim=0, rope_freq_base=10000.0, rope_half=True, window=0, out_gate=False, n_ff=0,
                 ff_act=FF_SILU, ff_bias=False) -> LayerConfig:
    return LayerConfig(mixer=MIXER_LATENT, n_head=n_head, n_head_kv=1, key_dim=key_dim, value_dim=value_dim, rope_dim=rope_dim,
                       rope_freq_base=rope_freq_base, attn_scale=scale, window=window, kv_from=-1, n_ff=n_ff, rope_half=int(rope_half),
                       kv_rank=kv_rank, out_gate=int(out_gate), ff_act=ff_act, ff_bias=int(ff_bias))


def delta_layer(n_head, n_head_kv, key_dim, value_dim, conv_taps, n_ff=0, ff_act=FF_SILU, ff_bias=False) -> LayerConfig:
    return LayerConfig(mixer=MIXER_DELTA, n_head=n_head, n_head_kv=n_head_kv, key_dim=key_dim, value_dim=value_dim, conv_taps=conv_taps,
                       kv_from=-1, n_ff=n_ff, ff_act=ff_act, ff_bias=int(ff_bias))


def config(n_layer, n_embd, n_vocab, n_ctx, eps, kv_block=16) -> el.Config:
    c = el.Config()
    c.n_layer, c.n_embd, c.n_vocab, c.n_ctx, c.rms_eps, c.kv_block, c.shard_count = n_layer, n_embd, n_vocab, n_ctx, eps, kv_block, 1
    return c


def _array(layers):
    arr = (LayerConfig * len(layers))()
    for i, l in enumerate(layers):
        arr[i] = l
    return arr


def check_layers(cfg: el.Config, layers, st: StackConfig | None = None) -> int:
    return int(eb.lib().emelb_llama_check_stack(C.byref(cfg), C.byref(st or stack()), _array(layers)))


def in_rows(l: LayerConfig) -> int:
    """Rows of the stacked input projections."""
    if l.mixer == MIXER_LINEAR:
        return 2 * l.n_head * (l.key_dim + l.value_dim)
    if l.mixer == MIXER_LATENT:
        return l.n_head * (l.key_dim + l.rope_dim + (l.value_dim if l.out_gate else 0)) + l.kv_rank + l.rope_dim
    if l.mixer == MIXER_DELTA:
        return 2 * l.n_head_kv * l.key_dim + 2 * l.n_head * l.value_dim + 2 * l.n_head
    return l.n_head * l.key_dim + (l.n_head_kv * (l.key_dim + l.value_dim) if l.kv_from < 0 else 0)


def side_by_side(o: np.ndarray, down: np.ndarray) -> np.ndarray:
    """The matrix of LAYER_OUT: output projection (columns padded to a multiple of 8) and down projection."""
    out = np.zeros((o.shape[0], pad8(o.shape[1]) + down.shape[1]), o.dtype)
    out[:, :o.shape[1]] = o
    out[:, pad8(o.shape[1]):] = down
    return out


class Session(el.Session):
    """An el.Session over layers; float32 = every operand and cache in f32."""

    def __init__(self, backend: eb.Backend, cfg: el.Config, layers, float32: bool = False, st: StackConfig | None = None):
        self.be, self.cfg, self.layers, self.stack = backend, cfg, list(layers), st or stack()
        self.n_runs = len(self.layers) + max(0, self.stack.loop_times - 1) * (self.stack.loop_stop - self.stack.loop_start)
        self._h = C.c_void_p()
        self._tensors, self._keep = [], []
        err = eb.lib().emelb_llama_create_stack(backend.handle, C.byref(cfg), C.byref(self.stack), _array(self.layers), 1 if float32 else 0,
                                                C.byref(self._h))
        if err != eb.OK:
            raise eb.BackendError(f"emelb_llama_create_stack failed with error mask {err}")
        self.last_error = eb.OK

    def close(self):
        super().close()
        for t in self._tensors:
            self.be.evict(t)
        self._tensors, self._keep = [], []

    def _upload(self, host: np.ndarray, t: int) -> int:
        # residency ids above the ones files' tensors get, never used twice on a backend
        tensor_id = getattr(self.be, "next_layered_tensor", 1 << 24)
        self.be.next_layered_tensor = tensor_id + 1
        dev = self.be.upload(tensor_id, host, tensor_type=t)
        self._tensors.append(tensor_id)
        self._keep.append(host)   # its address is the residency key
        return dev

    def _bind(self, layer, role, view) -> bool:
        return self._ret(eb.lib().emelb_llama_bind(self._h, layer, role, C.byref(view)))

    def bind_matrix_at(self, layer: int, role: int, dev: int, rows: int, k: int, ld: int) -> bool:
        """A bf16 matrix already on the device; ld elements between rows."""
        return self._bind(layer, role, eb.strided_view(dev, eb.BF16, [k, rows, 1, 1], [2, 2 * ld, 2 * ld * rows, 2 * ld * rows]))

    def bind_vector_at(self, layer: int, role: int, dev: int, n: int, rows: int = 1) -> bool:
        return self._bind(layer, role, eb.strided_view(dev, eb.F32, [n, rows, 1, 1], [4, 4 * n, 4 * n * rows, 4 * n * rows]))

    def load_matrix(self, layer: int, role: int, bits: np.ndarray, also=()) -> bool:
        """bits: bf16 bit patterns [rows, k]; rows are padded to 16 bytes.  also: further (layer, role) the same matrix serves."""
        rows, k = bits.shape
        ld = pad8(k)
        host = np.zeros((rows, ld), np.uint16)
        host[:, :k] = bits
        dev = self._upload(host, eb.BF16)
        return all(self.bind_matrix_at(i, r, dev, rows, k, ld) for i, r in [(layer, role), *also])

    def load_vector(self, layer: int, role: int, values: np.ndarray) -> bool:
        host = np.array(values, np.float32, order="C", copy=True)
        rows, n = (1, host.shape[0]) if host.ndim == 1 else host.shape
        return self.bind_vector_at(layer, role, self._upload(host, eb.F32), n, rows)

    def trace_layers(self, max_tokens: int):
        """Array the following prompt batches write their residual streams to ({layer runs, tokens, n_embd} packed at
        its start); 0 turns it off."""
        self._trace = np.zeros((self.n_runs, max(max_tokens, 1), self.cfg.n_embd), np.float32)
        self._ret(eb.lib().emelb_llama_trace_layers(self._h, self._trace.ctypes.data if max_tokens else None, max_tokens))
        return self._trace
