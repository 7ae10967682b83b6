"""Layered decoder sessions (include/emelb_llama.h, emelb_llama_create_layers): a decoder described layer by layer,
stepped through the same session calls as the block-quantized one."""
from __future__ import annotations

import ctypes as C

import numpy as np

import emel_cpp_b200 as eb
from emel_cpp_b200 import llama as el

MIXER_ATTENTION, MIXER_LINEAR = 0, 1
(MIX_IN, MIX_CONV, MIX_NORM_Q, MIX_NORM_K, MIX_HEADS, MIX_NORM_OUT, FFN_IN, FFN_IN_BIAS, FFN_DOWN_BIAS) = range(12, 21)


class LayerConfig(C.Structure):
    _fields_ = [("mixer", C.c_int32), ("n_head", C.c_int32), ("n_head_kv", C.c_int32), ("key_dim", C.c_int32),
                ("value_dim", C.c_int32), ("conv_taps", C.c_int32), ("norm_qk", C.c_int32), ("norm_v", C.c_int32),
                ("mix_heads", C.c_int32), ("rope_dim", C.c_int32), ("rope_freq_base", C.c_float),
                ("attn_scale", C.c_float), ("window", C.c_int32), ("keep_first", C.c_int32), ("kv_from", C.c_int32),
                ("n_ff", C.c_int32), ("decay", C.POINTER(C.c_float))]


def linear_layer(n_head, key_dim, value_dim, decay, n_ff=0) -> LayerConfig:
    if len(decay) != n_head:
        raise ValueError(f"{len(decay)} decays for {n_head} heads")
    l = LayerConfig(mixer=MIXER_LINEAR, n_head=n_head, key_dim=key_dim, value_dim=value_dim, kv_from=-1, n_ff=n_ff)
    l._decay = (C.c_float * n_head)(*[float(d) for d in decay])   # alive as long as the description
    l.decay = C.cast(l._decay, C.POINTER(C.c_float))
    return l


def attention_layer(n_head, n_head_kv, key_dim, value_dim, scale, conv_taps=0, norm_qk=True, norm_v=True, mix_heads=True,
                    rope_dim=0, rope_freq_base=10000.0, window=0, keep_first=0, kv_from=-1, n_ff=0) -> LayerConfig:
    return LayerConfig(mixer=MIXER_ATTENTION, n_head=n_head, n_head_kv=n_head_kv, key_dim=key_dim, value_dim=value_dim,
                       conv_taps=conv_taps, norm_qk=int(norm_qk), norm_v=int(norm_v), mix_heads=int(mix_heads),
                       rope_dim=rope_dim, rope_freq_base=rope_freq_base, attn_scale=scale, window=window,
                       keep_first=keep_first, kv_from=kv_from, n_ff=n_ff)


def config(n_layer, n_embd, n_vocab, n_ctx, eps, kv_block=16) -> el.Config:
    c = el.Config()
    c.n_layer, c.n_embd, c.n_vocab, c.n_ctx, c.rms_eps, c.kv_block, c.shard_count = n_layer, n_embd, n_vocab, n_ctx, eps, kv_block, 1
    return c


def _array(layers):
    arr = (LayerConfig * len(layers))()
    for i, l in enumerate(layers):
        arr[i] = l
    return arr


def check_layers(cfg: el.Config, layers) -> int:
    return int(eb.lib().emelb_llama_check_layers(C.byref(cfg), _array(layers)))


def in_rows(l: LayerConfig) -> int:
    """Rows of the stacked input projections."""
    if l.mixer == MIXER_LINEAR:
        return 2 * l.n_head * (l.key_dim + l.value_dim)
    return l.n_head * l.key_dim + (l.n_head_kv * (l.key_dim + l.value_dim) if l.kv_from < 0 else 0)


class Session(el.Session):
    """An el.Session over layers; float32 = every operand and cache in f32."""

    def __init__(self, backend: eb.Backend, cfg: el.Config, layers, float32: bool = False):
        self.be, self.cfg, self.layers = backend, cfg, list(layers)
        self._h = C.c_void_p()
        self._tensors, self._keep = [], []
        err = eb.lib().emelb_llama_create_layers(backend.handle, C.byref(cfg), _array(self.layers), 1 if float32 else 0, C.byref(self._h))
        if err != eb.OK:
            raise eb.BackendError(f"emelb_llama_create_layers failed with error mask {err}")
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

    def load_matrix(self, layer: int, role: int, bits: np.ndarray) -> bool:
        """bits: bf16 bit patterns [rows, k]; rows are padded to 16 bytes."""
        rows, k = bits.shape
        ld = (k + 7) // 8 * 8
        host = np.zeros((rows, ld), np.uint16)
        host[:, :k] = bits
        return self.bind_matrix_at(layer, role, self._upload(host, eb.BF16), rows, k, ld)

    def load_vector(self, layer: int, role: int, values: np.ndarray) -> bool:
        host = np.array(values, np.float32, order="C", copy=True)
        rows, n = (1, host.shape[0]) if host.ndim == 1 else host.shape
        return self.bind_vector_at(layer, role, self._upload(host, eb.F32), n, rows)

    def trace_layers(self, max_tokens: int):
        """Array the following prompt batches write their residual streams to ({n_layer, tokens, n_embd} packed at its
        start); 0 turns it off."""
        self._trace = np.zeros((self.cfg.n_layer, max(max_tokens, 1), self.cfg.n_embd), np.float32)
        self._ret(eb.lib().emelb_llama_trace_layers(self._h, self._trace.ctypes.data if max_tokens else None, max_tokens))
        return self._trace
