"""The Sikivik decoder: configuration and tensor names, mapped onto the block decoder (decoder.BlockDecoder).

A model is a folder with config.json and model.safetensors. config.json lists the layers; each has a mixer
('attention': sliding-window softmax attention with short convolutions on q / k / v, value mixing and a
sigmoid output gate; 'gla': gated linear attention; 'retention') beside a silu-gated feed-forward that reads
the same normed row. Layer i's tensors are 'l<i>.norm1', 'l<i>.mix.*' and 'l<i>.mlp.*'; 'embed', 'final.norm'
and 'head' complete the model. Nothing here is tied to particular sizes: they are read.
"""
from __future__ import annotations

from typing import List, Optional

import numpy as np

from . import api
from .decoder import BlockConfig, BlockDecoder, BlockTensors, MIXER_ATTENTION, MIXER_RECURRENT
from .safetensors import SafetensorsFile


class ConfigError(api.TensorError):
    pass


def block_config(layer: dict, decay_rank: int = 0) -> BlockConfig:
    """One entry of config.json's 'layers'. decay_rank: rows of the 'gla' gate's first matrix (a tensor's shape)."""
    m, kind = layer["mixer"], layer["type"]
    mlp = layer.get("mlp")
    if mlp is not None and mlp.get("kind", "dense") != "dense":
        raise ConfigError(f"unknown feed-forward '{mlp['kind']}'")
    rot = m.get("rot") or {"base": 1.0, "dims": 0}
    b = BlockConfig(heads=m["heads"], dim=m["dim"], vdim=m["vdim"], ffn=0 if mlp is None else mlp["ff"],
                    rot_dims=rot["dims"], rot_base=float(rot["base"]))
    if kind == "attention":
        b.mixer, b.kv_heads, b.scale = MIXER_ATTENTION, m["kv_heads"], float(m["scale"])
        b.window = (m.get("mask") or {}).get("size") or 0
        b.conv_taps, b.value_mix, b.out_gate = m.get("conv") or 0, bool(m.get("v_mix")), True
    elif kind == "gla":
        b.mixer, b.q_scale = MIXER_RECURRENT, b.dim ** -0.5
        b.decay_rank, b.decay_tau = decay_rank, float(m["tau"])
    elif kind == "retention":
        b.mixer, b.k_scale = MIXER_RECURRENT, b.dim ** -0.5
        if len(m["decay"]) != b.heads:
            raise ConfigError(f"{len(m['decay'])} decays for {b.heads} heads")
    else:
        raise ConfigError(f"unknown mixer '{kind}'")
    return b


def block_tensors(f: SafetensorsFile, i: int, layer: dict) -> BlockTensors:
    """The tensors of layer i in the block decoder's terms (matrices as bf16 bit patterns, the rest f32)."""
    mix, mlp, m = f"l{i}.mix.", f"l{i}.mlp.", layer["mixer"]
    t = BlockTensors(norm=f.f32(f"l{i}.norm1"), q=f.bf16(mix + "q"), k=f.bf16(mix + "k"), v=f.bf16(mix + "v"),
                     g=f.bf16(mix + "g"), o=f.bf16(mix + "o"))
    if layer["type"] == "attention":
        t.q_bias, t.k_bias, t.v_bias, t.o_bias = (f.f32(mix + n + ".b") for n in "qkvo")
        if m.get("conv"):
            t.conv = np.concatenate([f.f32(mix + n + ".conv") for n in "qkv"])
        if m.get("v_mix"):
            t.value_lambda = float(f.f32(mix + "vmix").reshape(()))
    elif layer["type"] == "gla":
        t.a1, t.decay_w, t.decay_b = f.bf16(mix + "a1"), f.f32(mix + "a2"), f.f32(mix + "a2.b")
        t.head_norm = f.f32(mix + "norm")
    else:
        t.decay = np.asarray(m["decay"], np.float32)
    if layer.get("mlp") is not None:
        t.gate, t.up, t.down = (f.bf16(mlp + n) for n in ("gate", "up", "down"))
    return t


def load(config: dict, weights_path: str, backend: Optional[api.Backend] = None, *, max_seq: int, act_dtype: int = api.BF16,
         block_rows: int = 0) -> BlockDecoder:
    f = SafetensorsFile(weights_path)
    layers: List[dict] = config["layers"]
    blocks = [block_config(L, f.info(f"l{i}.mix.a1").shape[0] if L["type"] == "gla" else 0) for i, L in enumerate(layers)]
    dec = BlockDecoder(backend or api.gpu_backend(), hidden=config["width"], vocab=config["vocab"], blocks=blocks, max_seq=max_seq,
                       rms_eps=float(config["norm"]["eps"]), act_dtype=act_dtype, block_rows=block_rows)
    for i, L in enumerate(layers):
        dec.set_block(i, block_tensors(f, i, L))
    dec.set_head(f.bf16("embed"), f.f32("final.norm"), f.bf16("head"))
    return dec

