"""Plain, slow restatement (numpy) of the decoders whose layers each name their own mixer: windowed
attention with short convolutions, value mixing and an output gate; gated linear attention; retention.
One function per mechanism, written from the equations, every sequence from its first token with
explicit loops over positions and no cache. Test infrastructure: nothing in the product imports it
and it imports nothing of the product.

Conventions: a row per token; T tokens, D model width. `cfg` is the model's config.json as a dict,
`w` maps tensor names to float arrays. `dt` is the arithmetic type (float64 by default).

    layer      x <- x + mixer(h) + ff(h),  h = norm(x)                  (one norm, both read it)
    attention  q, k, v = conv(W h + b); rotate q, k; v <- (1 - l) v + l v_first
               o_i = sum_{i-W < j <= i} softmax_j(scale q_i . k_j) v_j;  W_o (o * sigmoid(W_g h)) + b_o
    gla        S_t = diag(a_t) S_{t-1} + k_t v_t^T,  o_t = S_t^T q_t,  a_t = sigmoid(W_2 W_1 h + b)^(1/tau)
    retention  S_t = d S_{t-1} + k_t v_t^T,          o_t = S_t^T q_t   (q, k rotated, d fixed per head)
"""
from __future__ import annotations

import json
import struct

import numpy as np


def bf16_to_f32(u16):
    return (np.asarray(u16, dtype=np.uint16).astype(np.uint32) << 16).view(np.float32)


def read_model(folder):
    """config.json and the tensors of model.safetensors (bf16 / f32 / i32) of a folder."""
    with open(f"{folder}/config.json") as f:
        cfg = json.load(f)
    with open(f"{folder}/model.safetensors", "rb") as f:
        raw = f.read()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, t in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = t["data_offsets"]
        data = raw[8 + n + a:8 + n + b]
        if t["dtype"] == "BF16":
            v = bf16_to_f32(np.frombuffer(data, np.uint16))
        else:
            v = np.frombuffer(data, {"F32": np.float32, "I32": np.int32}[t["dtype"]])
        out[name] = v.reshape(t["shape"])
    return cfg, out


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def causal_conv(u, taps):
    """y_t[c] = sum_j taps[c, j] u_{t - n + 1 + j}[c]; rows before the first are zero."""
    n = taps.shape[1]
    y = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * u[s]
    return y


def rotate_half(x, base, dims, positions):
    """Rotation of the pairs (i, i + dims / 2), i < dims / 2, of the last axis by p * base^(-2i / dims).
    x [T, heads, d]."""
    y = x.copy()
    half = dims // 2
    for i in range(half):
        a = positions * (float(base) ** (-2.0 * i / dims))
        c, s = np.cos(a)[:, None].astype(x.dtype), np.sin(a)[:, None].astype(x.dtype)
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i] = u * c - v * s
        y[:, :, i + half] = v * c + u * s
    return y


def window_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, e]; position i sees j with 0 <= i - j < window (None: all earlier)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    for i in range(T):
        lo = 0 if window is None else max(0, i - window + 1)
        for h in range(H):
            g = h // (H // G)
            s = (k[lo:i + 1, g] @ q[i, h]) * scale
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, g]
    return out


def decayed_state(q, k, v, decay):
    """S_t = diag(decay_t) S_{t-1} + k_t v_t^T, o_t = S_t^T q_t per head. q, k, decay [T, H, d], v [T, H, e].
    Returns (o [T, H, e], last S [H, d, e])."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]), q.dtype)
    o = np.zeros((T, H, v.shape[2]), q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = decay[t, h][:, None] * S[h] + np.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def mixer_attention(m, w, h, vfirst, is_first, dt):
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w[n].T + w[n + ".b"] for n in "qkv")
    if m.get("conv"):
        q, k, v = (causal_conv(u, w[n + ".conv"]) for u, n in ((q, "q"), (k, "k"), (v, "v")))
    pos = np.arange(T, dtype=np.float64)
    q, k, v = q.reshape(T, H, d), k.reshape(T, G, d), v.reshape(T, G, e)
    if m.get("rot"):
        q = rotate_half(q, m["rot"]["base"], m["rot"]["dims"], pos)
        k = rotate_half(k, m["rot"]["base"], m["rot"]["dims"], pos)
    if m.get("v_mix"):
        if is_first:
            vfirst = v
        else:
            lam = dt(w["vmix"].reshape(()))
            v = (1 - lam) * v + lam * vfirst
    o = window_attention(q, k, v, dt(m["scale"]), m["mask"]["size"] if m.get("mask") else None)
    o = o.reshape(T, H * e) * sigmoid(h @ w["g"].T)
    return o @ w["o"].T + w["o.b"], vfirst


def gla_decay(h, a1, a2, b, tau):
    z = (h @ a1.T) @ a2.T + b
    return np.exp(-np.logaddexp(0.0, -z) / tau)   # sigmoid(z)^(1 / tau)


def mixer_gla(m, w, h, eps, dt):
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).reshape(T, H, d) * dt(d) ** dt(-0.5)
    k = (h @ w["k"].T).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, e)
    a = gla_decay(h, w["a1"], w["a2"], w["a2.b"], dt(m["tau"])).reshape(T, H, d)
    o, _ = decayed_state(q, k, v, a)
    o = (rms(o, eps) * w["norm"]).reshape(T, H * e) * silu(h @ w["g"].T)
    return o @ w["o"].T


def mixer_retention(m, w, h, eps, dt):
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    pos = np.arange(T, dtype=np.float64)
    q = rotate_half((h @ w["q"].T).reshape(T, H, d), m["rot"]["base"], m["rot"]["dims"], pos)
    k = rotate_half((h @ w["k"].T).reshape(T, H, d), m["rot"]["base"], m["rot"]["dims"], pos) * dt(d) ** dt(-0.5)
    v = (h @ w["v"].T).reshape(T, H, e)
    a = np.broadcast_to(np.asarray(m["decay"], dt)[None, :, None], q.shape)
    o, _ = decayed_state(q, k, v, a)
    o = rms(o, eps).reshape(T, H * e) * silu(h @ w["g"].T)
    return o @ w["o"].T


def feed_forward(w, h):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def forward(cfg, tensors, tokens, dt=np.float64, trace=None):
    """Logits [T, vocab] of one sequence; `trace`, if a list, receives the residual stream after every layer."""
    eps = dt(cfg["norm"]["eps"])
    w = {n: t.astype(dt) for n, t in tensors.items()}
    x = w["embed"][np.asarray(tokens)]
    vfirst, seen = None, False
    for i, L in enumerate(cfg["layers"]):
        mw = {n[len(f"l{i}.mix."):]: t for n, t in w.items() if n.startswith(f"l{i}.mix.")}
        fw = {n[len(f"l{i}.mlp."):]: t for n, t in w.items() if n.startswith(f"l{i}.mlp.")}
        h = rms(x, eps) * w[f"l{i}.norm1"]
        m = L["mixer"]
        if L["type"] == "attention":
            y, vfirst = mixer_attention(m, mw, h, vfirst, bool(m.get("v_mix")) and not seen, dt)
            seen = seen or bool(m.get("v_mix"))
        elif L["type"] == "gla":
            y = mixer_gla(m, mw, h, eps, dt)
        elif L["type"] == "retention":
            y = mixer_retention(m, mw, h, eps, dt)
        else:
            raise ValueError(L["type"])
        if L.get("mlp"):
            y = y + feed_forward(fw, h)
        x = x + y
        if trace is not None:
            trace.append(x.copy())
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T
