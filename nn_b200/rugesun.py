"""The Rugesun decoder: configuration and tensor names, mapped onto the block decoder (decoder.BlockDecoder).

A model is a folder with config.json and model.safetensors. Every layer is two sequential sublayers with a layer norm
behind each sum: attention through a latent over a sliding window (a layer with 'kv_from' reads an earlier layer's
latents), then a gelu-gated feed-forward, a mixture of silu-gated experts, or nothing. So a layer is one or two
blocks. Layer i's tensors are 'l<i>.norm1', 'l<i>.norm2', 'l<i>.mix.*' and 'l<i>.mlp.*'; 'embed', 'bigram' (the hashed
embedding of token pairs), 'final.norm' and 'head' complete the model. Nothing here is tied to particular sizes: they
are read.
"""
from __future__ import annotations

from typing import List, Optional, Tuple

from . import api
from .decoder import ACT_GELU_TANH, BlockConfig, BlockDecoder, BlockTensors, MIXER_LATENT, MIXER_NONE
from .safetensors import SafetensorsFile
from .sikivik import ConfigError


def layer_blocks(config: dict) -> List[Tuple[int, str, BlockConfig]]:
    """The blocks of the model in order: (layer, 'mix' or 'mlp', configuration)."""
    alpha, out, first = float(config["postln_alpha"]), [], {}
    for i, layer in enumerate(config["layers"]):
        if layer["type"] != "latent_attention":
            raise ConfigError(f"unknown mixer '{layer['type']}'")
        m, source = layer["mixer"], layer["mixer"].get("kv_from")
        if source is not None and (source not in first or config["layers"][source]["mixer"].get("kv_from") is not None):
            raise ConfigError(f"layer {i} reads the latents of layer {source}, which has none of its own in front of it")
        rot = m.get("rot") or {"base": 1.0, "dims": m["rot_dim"]}
        if rot["dims"] != m["rot_dim"]:
            raise ConfigError(f"layer {i}: {rot['dims']} of {m['rot_dim']} dimensions rotated")
        first[i] = len(out)
        out.append((i, "mix", BlockConfig(mixer=MIXER_LATENT, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], rot_dims=m["rot_dim"], rot_base=float(rot["base"]),
                                          scale=float(m["scale"]), window=(m.get("mask") or {}).get("size") or 0, post_norm=True, alpha=alpha,
                                          q_rank=m["q_rank"], kv_rank=m["kv_rank"], kv_from=-1 if source is None else first[source])))
        f = layer.get("mlp")
        if f is None:
            continue
        b = BlockConfig(mixer=MIXER_NONE, post_norm=True, alpha=alpha)
        kind = f.get("kind", "dense")
        if kind == "dense":
            b.ffn, b.ffn_act = f["ff"], ACT_GELU_TANH
        elif kind == "moe":
            b.experts, b.top, b.expert_ffn = f["router"]["experts"], f["router"]["top"], f["expert"]["ff"]
        else:
            raise ConfigError(f"unknown feed-forward '{kind}'")
        out.append((i, "mlp", b))
    return out


def block_tensors(f: SafetensorsFile, i: int, part: str, b: BlockConfig) -> BlockTensors:
    """The tensors of a block in the block decoder's terms (matrices as bf16 bit patterns, the rest f32)."""
    norm, p = f"l{i}.norm1" if part == "mix" else f"l{i}.norm2", f"l{i}.{part}."
    t = BlockTensors(norm=f.f32(norm), norm_bias=f.f32(norm + ".b"))
    if part == "mix":
        t.dq, t.uq, t.uk, t.uv, t.o = (f.bf16(p + n) for n in ("dq", "uq", "uk", "uv", "o"))
        t.q_norm = f.f32(p + "dq.norm")
        if b.kv_from < 0:
            t.dkv, t.kv_norm = f.bf16(p + "dkv"), f.f32(p + "dkv.norm")
    elif b.experts:
        t.router, t.router_bias = f.f32(p + "router"), f.f32(p + "router.b")
        t.expert = lambda e: tuple(f.bf16(f"{p}e{e}.{n}") for n in ("gate", "up", "down"))
    else:
        t.gate, t.up, t.down = (f.bf16(p + n) for n in ("gate", "up", "down"))
    return t


def load(config: dict, weights_path: str, backend: Optional[api.Backend] = None, *, max_seq: int, act_dtype: int = api.BF16,
         block_rows: int = 0) -> BlockDecoder:
    f = SafetensorsFile(weights_path)
    parts = layer_blocks(config)
    dec = BlockDecoder(backend or api.gpu_backend(), hidden=config["width"], vocab=config["vocab"], blocks=[b for _, _, b in parts], max_seq=max_seq,
                       rms_eps=float(config["norm"]["eps"]), act_dtype=act_dtype, block_rows=block_rows)
    for k, (i, part, b) in enumerate(parts):
        dec.set_block(k, block_tensors(f, i, part, b))
    pairs = (config.get("embedding") or {}).get("bigram")
    extra = {} if not pairs else dict(pair_table=f.bf16("bigram"), pair_mul=(pairs["mul_prev"], pairs["mul_cur"]))
    if pairs and f.info("bigram").shape[0] != pairs["buckets"] + 1:
        raise ConfigError(f"{f.info('bigram').shape[0]} rows for {pairs['buckets']} buckets")
    dec.set_head(f.bf16("embed"), f.f32("final.norm"), f.bf16("head"), final_norm_bias=f.f32("final.norm.b"),
                 logit_cap=float(config.get("logit_softcap") or 0.0), **extra)
    return dec
