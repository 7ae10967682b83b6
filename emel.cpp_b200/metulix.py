"""The Metulix design: decoder layers whose mixers are linear attention with a fixed decay per head ("lightning") or
windowed softmax attention with a short convolution, query / key / value norms, mixed heads and, optionally, another
layer's keys and values.  A model is a folder with config.json and model.safetensors."""
from __future__ import annotations

import json
import os

import numpy as np

import emel_cpp_b200 as eb
from emel_cpp_b200 import layered as ly
from emel_cpp_b200 import llama as el
from emel_cpp_b200 import safetensors as st

ARCHITECTURE = "Metulix"


def layer_configs(cfg: dict):
    out = []
    for i, layer in enumerate(cfg["layers"]):
        m, mlp = layer["mixer"], layer.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        ff = int(mlp["ff"]) if mlp else 0
        if layer["type"] == "lightning":
            out.append(ly.linear_layer(m["heads"], m["dim"], m["vdim"], m["decay"], n_ff=ff))
        elif layer["type"] == "attention":
            rot, mask, kv_from = m.get("rot") or {}, m.get("mask") or {}, m.get("kv_from")
            out.append(ly.attention_layer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], conv_taps=m.get("conv") or 0,
                                          rope_dim=rot.get("dims", 0), rope_freq_base=rot.get("base", 10000.0),
                                          window=mask.get("size") or 0, keep_first=mask.get("keep_first") or 0,
                                          kv_from=-1 if kv_from is None else kv_from, n_ff=ff))
        else:
            raise ValueError(f"layer {i}: mixer {layer['type']!r}")
    return out


def session_config(cfg: dict, n_ctx: int) -> el.Config:
    return ly.config(len(cfg["layers"]), cfg["width"], cfg["vocab"], n_ctx, cfg["norm"]["eps"])


def load(backend: eb.Backend, path: str, n_ctx: int = 4096, float32: bool = False) -> ly.Session:
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    return load_tensors(backend, cfg, st.File(os.path.join(path, "model.safetensors")), n_ctx, float32)


def load_tensors(backend: eb.Backend, cfg: dict, f: st.File, n_ctx: int, float32: bool = False) -> ly.Session:
    """Uploads and binds every tensor; a layer's input projections and its gate and up projections are stacked."""
    layers = layer_configs(cfg)
    sess = ly.Session(backend, session_config(cfg, n_ctx), layers, float32)

    def matrix(layer, role, *names):
        if not sess.load_matrix(layer, role, np.concatenate([f.bf16(n) for n in names])):
            raise ValueError(f"tensor {'|'.join(names)} does not fit the configuration")

    def vector(layer, role, *names):
        if not sess.load_vector(layer, role, np.concatenate([f.f32(n) for n in names])):
            raise ValueError(f"tensor {'|'.join(names)} does not fit the configuration")

    try:
        matrix(-1, el.TOKEN_EMBD, "embed")
        vector(-1, el.OUTPUT_NORM, "final.norm")
        matrix(-1, el.OUTPUT, "head")
        for i, l in enumerate(layers):
            p, mix, mlp = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            if l.mixer == ly.MIXER_LINEAR:
                matrix(i, ly.MIX_IN, mix + "q", mix + "k", mix + "v", mix + "g")
                vector(i, ly.MIX_NORM_OUT, mix + "norm")
            else:
                parts = ["q", "k", "v"] if l.kv_from < 0 else ["q"]
                matrix(i, ly.MIX_IN, *[mix + n for n in parts])
                if l.conv_taps:
                    vector(i, ly.MIX_CONV, *[f"{mix}{n}.conv" for n in parts])
                vector(i, ly.MIX_NORM_Q, mix + "q.norm")
                if l.kv_from < 0:
                    vector(i, ly.MIX_NORM_K, mix + "k.norm")
                vector(i, ly.MIX_HEADS, mix + "talk")
            matrix(i, el.ATTN_OUT, mix + "o")
            vector(i, el.ATTN_NORM, p + "norm1")
            if l.n_ff:
                vector(i, el.FFN_NORM, p + "norm2")
                matrix(i, ly.FFN_IN, mlp + "gate", mlp + "up")
                vector(i, ly.FFN_IN_BIAS, mlp + "gate.b", mlp + "up.b")
                matrix(i, el.FFN_DOWN, mlp + "down")
                vector(i, ly.FFN_DOWN_BIAS, mlp + "down.b")
    except Exception:
        sess.close()
        raise
    return sess
