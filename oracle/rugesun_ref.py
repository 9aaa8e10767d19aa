"""Plain, slow restatement (numpy) of the Rugesun decoder: sequential sublayers with a layer norm behind each sum,
multi-head attention through a latent (keys and values are linear images of one normed vector per token, plus one
rotated key part that all heads share) over a sliding window, latents that later layers read from an earlier one,
gelu-gated feed-forwards and mixtures of experts, a hashed embedding of token pairs, capped logits. One function per
mechanism, written from the equations, every sequence from its first token, no cache. Test infrastructure: nothing
in the product imports it and it imports nothing of the product.

Conventions: a row per token; T tokens, D model width. `cfg` is the model's config.json as a dict, tensors are float
arrays by name. `dt` is the arithmetic type (float64 by default).

    x_0      = E[t_i] + B[(a t_{i-1} + b t_i) mod n],  B[n] for the first token
    layer    x <- LN_1(alpha x + mixer(x));  x <- LN_2(alpha x + ff(x))
    mixer    c_q = rms(W_dq x) g_q,  (q^u_h, q^r_h) = head h of W_uq c_q;  (l, r) = W_dkv x,  c = rms(l) g_c
             s_ij = scale ((q^u_hi . W_uk,h c_j) + (R_i q^r_hi . R_j r_j)),  0 <= i - j < window
             W_o concat_h(sum_j softmax_j(s_ij) W_uv,h c_j)
    experts  z = W_r x + b;  sum over the top z of softmax(top z)_e W_d,e (silu(W_g,e x) * W_u,e x)
    logits   cap tanh((W LN(x)) / cap)
"""
from __future__ import annotations

import numpy as np

from .hybrid_ref import read_model, rms, rotate_half, silu  # noqa: F401


def layer_norm(x, w, b, eps):
    d = x - x.mean(-1, keepdims=True)
    return d / np.sqrt((d * d).mean(-1, keepdims=True) + eps) * w + b


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def pair_rows(tokens, mul_prev, mul_cur, buckets):
    """Row of the pair table for every token; the first token of a sequence has the row behind the buckets."""
    return [buckets if i == 0 else (int(tokens[i - 1]) * int(mul_prev) + int(t) * int(mul_cur)) % int(buckets) for i, t in enumerate(tokens)]


def latent(m, w, x, eps):
    """Per token: the normed latent c [T, kv_rank] and the rotated shared key part [T, rot_dim]."""
    y = x @ w["dkv"].T
    n = m["kv_rank"]
    r = rotate_half(y[:, None, n:], m["rot"]["base"], m["rot"]["dims"], np.arange(len(x), dtype=np.float64))[:, 0]
    return rms(y[:, :n], eps) * w["dkv.norm"], r


def latent_queries(m, w, x, eps):
    """Unrotated and rotated query parts, [T, H, dim] and [T, H, rot_dim]."""
    q = ((rms(x @ w["dq"].T, eps) * w["dq.norm"]) @ w["uq"].T).reshape(len(x), m["heads"], m["dim"] + m["rot_dim"])
    return q[..., :m["dim"]], rotate_half(q[..., m["dim"]:], m["rot"]["base"], m["rot"]["dims"], np.arange(len(x), dtype=np.float64))


def latent_attention(m, w, x, kv, eps, dt):
    c, r = kv
    T, H = len(x), m["heads"]
    qu, qr = latent_queries(m, w, x, eps)
    k = (c @ w["uk"].T).reshape(T, H, m["dim"])
    v = (c @ w["uv"].T).reshape(T, H, m["vdim"])
    size = (m.get("mask") or {}).get("size")
    out = np.zeros((T, H, m["vdim"]), x.dtype)
    for i in range(T):
        lo = 0 if size is None else max(0, i - size + 1)
        for h in range(H):
            s = (k[lo:i + 1, h] @ qu[i, h] + r[lo:i + 1] @ qr[i, h]) * dt(m["scale"])
            p = np.exp(s - s.max())
            out[i, h] = (p / p.sum()) @ v[lo:i + 1, h]
    return out.reshape(T, -1) @ w["o"].T


def feed_forward(w, x, act):
    return (act(x @ w["gate"].T) * (x @ w["up"].T)) @ w["down"].T


def route(z, top):
    """Chosen experts (largest logits) and the softmax over their logits, [T, top] each."""
    idx = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    c = np.take_along_axis(z, idx, -1)
    p = np.exp(c - c.max(-1, keepdims=True))
    return idx, p / p.sum(-1, keepdims=True)


def mixture(w, x, experts, top):
    idx, p = route(x @ w["router"].T + w["router.b"], top)
    y = np.zeros_like(x)
    for e in range(experts):
        ew = {n: w[f"e{e}.{n}"] for n in ("gate", "up", "down")}
        t, s = np.nonzero(idx == e)
        if len(t):
            y[t] += p[t, s][:, None] * feed_forward(ew, x[t], silu)
    return y


def soft_cap(z, cap):
    return z if not cap else cap * np.tanh(z / cap)


def part(w, prefix):
    return {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}


def forward(cfg, tensors, tokens, dt=np.float64, trace=None):
    """Logits [T, vocab] of one sequence; `trace`, if a list, receives the residual stream after every layer."""
    eps, alpha = dt(cfg["norm"]["eps"]), dt(cfg["postln_alpha"])
    w = {n: t.astype(dt) for n, t in tensors.items()}
    x = w["embed"][np.asarray(tokens)]
    pairs = (cfg.get("embedding") or {}).get("bigram")
    if pairs:
        x = x + w["bigram"][pair_rows(tokens, pairs["mul_prev"], pairs["mul_cur"], pairs["buckets"])]
    kv = {}
    for i, L in enumerate(cfg["layers"]):
        m, mw, fw = L["mixer"], part(w, f"l{i}.mix."), part(w, f"l{i}.mlp.")
        src = m.get("kv_from", i)
        if src == i:
            kv[i] = latent(m, mw, x, eps)
        x = layer_norm(alpha * x + latent_attention(m, mw, x, kv[src], eps, dt), w[f"l{i}.norm1"], w[f"l{i}.norm1.b"], eps)
        f = L.get("mlp")
        if f:
            y = feed_forward(fw, x, gelu_tanh) if f["kind"] == "dense" else mixture(fw, x, f["router"]["experts"], f["router"]["top"])
            x = layer_norm(alpha * x + y, w[f"l{i}.norm2"], w[f"l{i}.norm2.b"], eps)
        if trace is not None:
            trace.append(x.copy())
    x = layer_norm(x, w["final.norm"], w["final.norm.b"], eps)
    return soft_cap(x @ w["head"].T, cfg.get("logit_softcap"))
