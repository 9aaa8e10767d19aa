"""Prefill and decode throughput of the Sikivik and Rugesun designs at sizes of real layers (random weights), beside a
Qwen3-shaped decoder of equal width, heads and feed-forward with unquantized bf16 weights. Used by
`bench.py --model sikivik | rugesun`; `python -m nn_b200.blockbench --once SIZE` issues one prompt pass and a few
decode steps of one model (a launch list under a profiler)."""
from __future__ import annotations

import argparse
import json
import time

import numpy as np

from . import api
from .decoder import (ACT_GELU_TANH, BlockConfig, BlockDecoder, BlockTensors, Decoder, DecoderConfig, MIXER_ATTENTION, MIXER_LATENT, MIXER_NONE,
                      MIXER_RECURRENT)
from .formats import QuantFormat
from .safetensors import bf16_to_f32

# layers: two periods of (attention, gla, gla, retention); Qwen3: as many layers of its own
SIZES = {
    "width 2048": dict(hidden=2048, ff=6144, heads=16, kv=4, rec_heads=8, rec_dim=128, rec_vdim=256, window=512, rank=16, vocab=32768),
    "width 4096": dict(hidden=4096, ff=12288, heads=32, kv=8, rec_heads=16, rec_dim=128, rec_vdim=256, window=1024, rank=16, vocab=32768),
}
PERIODS = 2
# Rugesun: two periods of (dense, experts, dense, experts on the latents of the layer in front); every layer's attention
# has the heads and the window of the size above
LATENT = {
    "width 2048": dict(dim=128, rot=64, vdim=128, q_rank=768, kv_rank=512, experts=32, top=4, expert_ff=768),
    "width 4096": dict(dim=128, rot=64, vdim=128, q_rank=1536, kv_rank=512, experts=32, top=4, expert_ff=1536),
}


def _bits(rng, *shape):
    """bf16 bit patterns of values +-(1 .. 2) / 128: sums over a few thousand terms stay of order one."""
    return (rng.integers(0, 1 << 16, shape, dtype=np.uint16) & np.uint16(0x807F)) | np.uint16(0x3C00)


def block_model(backend, z, max_seq, act_dtype=api.BF16, seed=0):
    D, F = z["hidden"], z["ff"]
    attn = BlockConfig(MIXER_ATTENTION, z["heads"], z["kv"], 128, 128, F, 128, 1e6, 128 ** -0.5, z["window"], 4, True, True)
    gla = BlockConfig(MIXER_RECURRENT, z["rec_heads"], 1, z["rec_dim"], z["rec_vdim"], F, q_scale=z["rec_dim"] ** -0.5, decay_rank=z["rank"], decay_tau=16.0)
    ret = BlockConfig(MIXER_RECURRENT, z["rec_heads"], 1, z["rec_dim"], z["rec_vdim"], F, z["rec_dim"], 1e6, k_scale=z["rec_dim"] ** -0.5)
    blocks = [attn, gla, gla, ret] * PERIODS
    dec = BlockDecoder(backend, hidden=D, vocab=z["vocab"], blocks=blocks, max_seq=max_seq, act_dtype=act_dtype)
    rng = np.random.default_rng(seed)
    for i, b in enumerate(blocks):
        at = b.mixer == MIXER_ATTENTION
        kvh = b.kv_heads if at else b.heads
        q, k, v, m = b.heads * b.dim, kvh * b.dim, kvh * b.vdim, b.heads * b.vdim
        t = BlockTensors(norm=np.ones(D, np.float32), q=_bits(rng, q, D), k=_bits(rng, k, D), v=_bits(rng, v, D), g=_bits(rng, m, D), o=_bits(rng, D, m),
                         gate=_bits(rng, F, D), up=_bits(rng, F, D), down=_bits(rng, D, F))
        if at:
            t.q_bias, t.k_bias, t.v_bias, t.o_bias = (np.full(n, 0.01, np.float32) for n in (q, k, v, D))
            t.conv, t.value_lambda = rng.standard_normal((q + k + v, 4)).astype(np.float32) * 0.5, 0.5
        elif b.decay_rank:
            t.a1, t.decay_w, t.decay_b = _bits(rng, b.decay_rank, D), rng.standard_normal((q, b.decay_rank)).astype(np.float32), np.ones(q, np.float32)
            t.head_norm = np.ones(b.vdim, np.float32)
        else:
            t.decay = (1.0 - 2.0 ** -np.linspace(5, 12, b.heads)).astype(np.float32)
        dec.set_block(i, t)
    e = _bits(rng, z["vocab"], D)
    dec.set_head(e, np.ones(D, np.float32), e)
    return dec


def rugesun_blocks(z, y):
    mix = dict(mixer=MIXER_LATENT, heads=z["heads"], dim=y["dim"], vdim=y["vdim"], rot_dims=y["rot"], rot_base=1e6, scale=(y["dim"] + y["rot"]) ** -0.5,
               window=z["window"], post_norm=True, alpha=1.5, q_rank=y["q_rank"], kv_rank=y["kv_rank"])
    dense = dict(mixer=MIXER_NONE, post_norm=True, alpha=1.5, ffn=z["ff"], ffn_act=ACT_GELU_TANH)
    moe = dict(mixer=MIXER_NONE, post_norm=True, alpha=1.5, experts=y["experts"], top=y["top"], expert_ffn=y["expert_ff"])
    out = []
    for _ in range(PERIODS):
        at = len(out)
        for k, f in enumerate((dense, moe, dense, moe)):
            out += [BlockConfig(**mix, kv_from=at + 4 if k == 3 else -1), BlockConfig(**f)]
    return out


def rugesun_model(backend, z, max_seq, act_dtype=api.BF16, seed=0):
    D, y = z["hidden"], z["latent"]
    blocks = rugesun_blocks(z, y)
    dec = BlockDecoder(backend, hidden=D, vocab=z["vocab"], blocks=blocks, max_seq=max_seq, rms_eps=1e-5, act_dtype=act_dtype)
    rng = np.random.default_rng(seed)
    one, zero = np.ones(D, np.float32), np.zeros(D, np.float32)
    experts = [(_bits(rng, y["expert_ff"], D), _bits(rng, y["expert_ff"], D), _bits(rng, D, y["expert_ff"])) for _ in range(y["experts"])]
    for i, b in enumerate(blocks):
        t = BlockTensors(norm=one, norm_bias=zero)
        if b.mixer == MIXER_LATENT:
            H = b.heads
            t.dq, t.uq, t.q_norm = _bits(rng, b.q_rank, D), _bits(rng, H * (b.dim + b.rot_dims), b.q_rank), np.ones(b.q_rank, np.float32)
            t.uk, t.uv, t.o = _bits(rng, H * b.dim, b.kv_rank), _bits(rng, H * b.vdim, b.kv_rank), _bits(rng, D, H * b.vdim)
            if b.kv_from < 0:
                t.dkv, t.kv_norm = _bits(rng, b.kv_rank + b.rot_dims, D), np.ones(b.kv_rank, np.float32)
        elif b.experts:
            t.router, t.expert = bf16_to_f32(_bits(rng, b.experts, D)), experts.__getitem__
        else:
            t.gate, t.up, t.down = _bits(rng, b.ffn, D), _bits(rng, b.ffn, D), _bits(rng, D, b.ffn)
        dec.set_block(i, t)
    e = _bits(rng, z["vocab"], D)
    dec.set_head(e, one, e, final_norm_bias=zero, logit_cap=30.0, pair_table=_bits(rng, 4097, D), pair_mul=(29, 13))
    return dec


def qwen3_model(backend, z, max_seq, act_dtype=api.BF16, seed=0):
    import torch
    D, F, H, G, n = z["hidden"], z["ff"], z["heads"], z["kv"], 4 * PERIODS
    dev = torch.device("cuda", backend.device)
    dec = Decoder(backend, DecoderConfig(hidden=D, n_heads=H, n_kv_heads=G, head_dim=128, ffn=F, n_layers=n, vocab=z["vocab"], max_seq=max_seq,
                                         rope_theta=1e6, act_dtype=act_dtype))
    rng = np.random.default_rng(seed)

    def w(rows, cols):
        raw = torch.from_numpy(_bits(rng, rows, cols).view(np.uint8).reshape(-1)).to(dev)
        return api.DeviceWeight.from_device(backend, QuantFormat.BF16_DENSE, raw, rows, cols)

    one, oned = np.ones(D, np.float32), np.ones(128, np.float32)
    for i in range(n):
        dec.set_layer(i, w(H * 128, D), w(G * 128, D), w(G * 128, D), w(D, H * 128), w(F, D), w(F, D), w(D, F), one, one, oned, oned)
    embed = torch.from_numpy(_bits(rng, z["vocab"], D).view(np.int16)).to(dev).view(torch.bfloat16)
    dec.set_head(embed, one, w(z["vocab"], D))
    return dec


def weight_bytes(name, z):
    """Bytes of the weights one decoded token streams (bf16, the vocabulary projection included)."""
    D, F = z["hidden"], z["ff"]
    if name == "rugesun":
        y, H, total = z["latent"], z["heads"], 0
        for b in rugesun_blocks(z, y):
            if b.mixer == MIXER_LATENT:
                total += D * b.q_rank + H * (b.dim + b.rot_dims) * b.q_rank + H * (b.dim + b.vdim) * b.kv_rank + D * H * b.vdim
                total += D * (b.kv_rank + b.rot_dims) if b.kv_from < 0 else 0
            else:
                total += 3 * D * (b.ffn or b.top * b.expert_ffn) + 2 * D * b.experts   # (the router is f32)
        return 2 * total + 2 * D * z["vocab"]
    if name == "qwen3":
        per = 2 * D * (2 * z["heads"] * 128 + 2 * z["kv"] * 128 + 3 * F) * 4
    else:
        a = 3 * z["heads"] * 128 + 2 * z["kv"] * 128 + 3 * F
        r = 2 * z["rec_heads"] * z["rec_dim"] + 3 * z["rec_heads"] * z["rec_vdim"] + 3 * F
        per = 2 * D * (a + 3 * r + 2 * z["rank"])
    return PERIODS * per + 2 * D * z["vocab"]


def product_flops(name, z):
    """Multiply-adds of the layers' products per prompt token, times two (chosen experts only)."""
    return weight_bytes(name, z) - 2 * z["hidden"] * z["vocab"]


def measure(backend, name, z, prompt, new_tokens, reps=5):
    import torch
    dev = torch.device("cuda", backend.device)
    dec = MODELS[name](backend, z, prompt + new_tokens + 16)
    ids = np.random.default_rng(7).integers(0, z["vocab"], prompt).tolist()
    st = torch.cuda.Stream(device=dev)
    for _ in range(3):
        dec.prefill(ids, 0, st)
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record(st)
    for _ in range(reps):
        dec.prefill(ids, 0, st)
    e1.record(st)
    st.synchronize()
    prefill = e0.elapsed_time(e1) * 1e-3 / reps
    with torch.cuda.stream(st):
        for _ in range(3):
            dec.step(st)
        st.synchronize()
        l0 = backend.launch_count()
        g = torch.cuda.CUDAGraph()
        with torch.cuda.graph(g, stream=st):
            dec.step(torch.cuda.current_stream())
        launches = backend.launch_count() - l0
        for _ in range(3):
            g.replay()
        e0.record(st)
        for _ in range(new_tokens):
            g.replay()
        e1.record(st)
        st.synchronize()
    backend.device_status(st)
    step = e0.elapsed_time(e1) * 1e-3 / new_tokens
    dec.release()
    for t in dec._keep:
        if isinstance(t, api.DeviceWeight):
            t.release()
    return {"prefill_tokens_per_s": prompt / prefill, "prefill_ms": prefill * 1e3, "prefill_product_tflops": product_flops(name, z) * prompt / prefill / 1e12,
            "decode_tokens_per_s": 1.0 / step, "decode_us_per_token": step * 1e6, "decode_weight_gbs": weight_bytes(name, z) / step / 1e9,
            "decode_launches": int(launches)}


MODELS = {"sikivik": block_model, "rugesun": rugesun_model, "qwen3": qwen3_model}


def run(prompt=4096, new_tokens=128, reps=5, model="sikivik", beside=("qwen3",)):
    backend = api.gpu_backend()
    out = {}
    for size in SIZES:
        z = dict(SIZES[size], latent=LATENT[size])
        r = out[size] = {n: measure(backend, n, z, prompt, new_tokens, reps) for n in (model, *beside)}
        for n in beside:
            r[f"{model}_over_{n}"] = {k: r[model][k] / r[n][k] for k in ("prefill_tokens_per_s", "decode_tokens_per_s")}
    return out


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--once", choices=sorted(SIZES))
    ap.add_argument("--which", default="sikivik", choices=sorted(MODELS))
    ap.add_argument("--prompt", type=int, default=1024)
    ap.add_argument("--new", type=int, default=2)
    a = ap.parse_args()
    if not a.once:
        print(json.dumps(run()))
        return
    b = api.gpu_backend()
    dec = MODELS[a.which](b, dict(SIZES[a.once], latent=LATENT[a.once]), a.prompt + a.new + 8)
    t0 = time.perf_counter()
    dec.prefill(np.random.default_rng(7).integers(0, SIZES[a.once]["vocab"], a.prompt).tolist(), 0, 0)
    for _ in range(a.new):
        dec.step(0)
    b.device_status(0)
    print(f"{a.which}, {a.once}: {a.prompt} prompt tokens and {a.new} steps in {time.perf_counter() - t0:.3f} s")


if __name__ == "__main__":
    main()
