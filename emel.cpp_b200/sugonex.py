"""The Sugonex design: parallel layers (mixer and feed-forward read the same stream, each behind its own RMS norm) whose mixers
are latent attention with a rotated part and an output gate, windowed latent attention without positions, or the gated
delta rule; some layers run several times with the same weights.  A model is a folder with config.json and
model.safetensors."""
from __future__ import annotations

import json
import os

import numpy as np

import emel_cpp_b200 as eb
from emel_cpp_b200 import layered as ly
from emel_cpp_b200 import llama as el
from emel_cpp_b200 import safetensors as st

ARCHITECTURE = "Sugonex"


def layer_configs(cfg: dict):
    out = []
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, kind = layer["mixer"], layer.get("mlp"), layer["type"]
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"layer {i}: feed-forward kind {mlp['kind']!r}")
        ff = dict(n_ff=int(mlp["ff"]) if mlp else 0, ff_act=ly.FF_GELU_TANH)
        window = (m.get("mask") or {}).get("size") or 0
        if kind == "latent_attention":
            rot = m.get("rot") or {}
            rot_dim = m.get("rot_dim") or 0
            if rot.get("dims", rot_dim) != rot_dim:
                raise ValueError(f"layer {i}: {rot['dims']} rotated dimensions in a part of {rot_dim}")
            out.append(ly.latent_layer(m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["scale"], rope_dim=rot_dim,
                                       rope_freq_base=rot.get("base", 10000.0), rope_half=True, window=window, out_gate=True, **ff))
        elif kind == "latent_attention_2":
            out.append(ly.latent_layer(m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["scale"], window=window, **ff))
        elif kind == "delta":
            out.append(ly.delta_layer(m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], **ff))
        else:
            raise ValueError(f"layer {i}: mixer {kind!r}")
    return out


def stack_config(cfg: dict) -> ly.StackConfig:
    loop = cfg.get("loop")
    return ly.stack(ly.STACK_PARALLEL, ly.NORM_RMS, loop=(loop["start"], loop["stop"], loop["times"]) if loop else None, loop_step=bool(loop),
                    logit_scale=1.0 if cfg.get("logit_scale") is None else cfg["logit_scale"], logit_softcap=cfg.get("logit_softcap") or 0.0)


def session_config(cfg: dict, n_ctx: int) -> el.Config:
    return ly.config(len(cfg["layers"]), cfg["width"], cfg["vocab"], n_ctx, cfg["norm"]["eps"])


def load(backend: eb.Backend, path: str, n_ctx: int = 4096, float32: bool = False) -> ly.Session:
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    return load_tensors(backend, cfg, st.File(os.path.join(path, "model.safetensors")), n_ctx, float32)


def load_tensors(backend: eb.Backend, cfg: dict, f: st.File, n_ctx: int, float32: bool = False) -> ly.Session:
    """Uploads and binds every tensor; projections of the same input are stacked, output and down projection of a layer
    are set side by side, and the norms of the stream, stored around zero, become plain weights."""
    layers = layer_configs(cfg)
    sess = ly.Session(backend, session_config(cfg, n_ctx), layers, float32, stack_config(cfg))

    def need(ok, *names):
        if not ok:
            raise ValueError(f"tensor {'|'.join(names)} does not fit the configuration")

    def matrix(layer, role, *names, also=()):
        need(sess.load_matrix(layer, role, np.concatenate([f.bf16(n) for n in names]), also), *names)

    def vector(layer, role, *names):
        need(sess.load_vector(layer, role, np.concatenate([f.f32(n) for n in names])), *names)

    def around_one(layer, role, name):
        need(sess.load_vector(layer, role, np.float32(1.0) + f.f32(name)), name)

    try:
        matrix(-1, el.TOKEN_EMBD, "embed", also=[(-1, el.OUTPUT)])
        around_one(-1, el.OUTPUT_NORM, "final.norm")
        if sess.stack.loop_step:
            vector(-1, ly.LOOP_STEP, "loop.step")
        for i, l in enumerate(layers):
            p, mix, mlp = f"l{i}.", f"l{i}.mix.", f"l{i}.mlp."
            if l.mixer == ly.MIXER_DELTA:
                matrix(i, ly.MIX_IN, *[mix + n for n in ("q", "k", "v", "g", "b", "a")])
                vector(i, ly.MIX_CONV, *[f"{mix}{n}.conv" for n in ("q", "k", "v")])
                vector(i, ly.MIX_DECAY_LOG, mix + "A_log")
                vector(i, ly.MIX_STEP_BIAS, mix + "dt_bias")
                vector(i, ly.MIX_NORM_OUT, mix + "norm")
            else:
                matrix(i, ly.MIX_IN, *[mix + n for n in (("q", "g", "dkv") if l.out_gate else ("q", "dkv"))])
                vector(i, ly.MIX_LATENT_NORM, mix + "dkv.norm")
                matrix(i, ly.MIX_LATENT_UP, mix + "uk", mix + "uv")
            around_one(i, el.ATTN_NORM, p + "norm1")
            if l.n_ff:
                around_one(i, el.FFN_NORM, p + "norm2")
                matrix(i, ly.FFN_IN, mlp + "gate", mlp + "up")
                need(sess.load_matrix(i, ly.LAYER_OUT, ly.side_by_side(f.bf16(mix + "o"), f.bf16(mlp + "down"))), mix + "o", mlp + "down")
            else:
                matrix(i, el.ATTN_OUT, mix + "o")
    except Exception:
        sess.close()
        raise
    return sess
