"""Small random Rugesun models for the tests: config.json dicts and tensors (f32 values that are exact in bf16); folders
are written by block_models.write_folder. Shares no code with the product."""
import numpy as np

from block_models import bf16_exact, write_folder  # noqa: F401

DENSE = {"kind": "dense", "ff": 90}


def moe(experts=6, top=2, ff=40):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def layer(heads=3, dim=24, rot_dim=8, vdim=20, q_rank=28, kv_rank=36, window=9, base=3e3, scale=0.23, kv_from=None, mlp=DENSE):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": window}, "scale": scale,
         "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(layers, width=72, vocab=150, eps=1e-5, alpha=1.7, cap=9.0, pairs=(61, 11, 5)):
    c = {"architecture": "Rugesun", "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha, "vocab": vocab, "width": width, "logit_softcap": cap}
    if pairs:
        c["embedding"] = {"bigram": {"buckets": pairs[0], "mul_prev": pairs[1], "mul_cur": pairs[2]}}
    return c


def tensors(cfg, seed=0):
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return bf16_exact(rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def around(n, mean, spread):
        return bf16_exact(mean + spread * rng.standard_normal(n))

    t = {"embed": bf16_exact(rng.standard_normal((V, D)))}
    if cfg.get("embedding"):
        t["bigram"] = bf16_exact(rng.standard_normal((cfg["embedding"]["bigram"]["buckets"] + 1, D)))
    for i, L in enumerate(cfg["layers"]):
        m, p, f = L["mixer"], f"l{i}.mix.", f"l{i}.mlp."
        H = m["heads"]
        t[p + "dq"], t[p + "dq.norm"] = mat(m["q_rank"], D), around(m["q_rank"], 1.0, 0.2)
        t[p + "uq"] = mat(H * (m["dim"] + m["rot_dim"]), m["q_rank"])
        if "kv_from" not in m:
            t[p + "dkv"], t[p + "dkv.norm"] = mat(m["kv_rank"] + m["rot_dim"], D), around(m["kv_rank"], 1.0, 0.2)
        t[p + "uk"], t[p + "uv"] = mat(H * m["dim"], m["kv_rank"]), mat(H * m["vdim"], m["kv_rank"])
        t[p + "o"] = mat(D, H * m["vdim"])
        names = ["norm1"]
        if L["mlp"]:
            names.append("norm2")
            if L["mlp"]["kind"] == "dense":
                F = L["mlp"]["ff"]
                t[f + "gate"], t[f + "up"], t[f + "down"] = mat(F, D), mat(F, D), mat(D, F)
            else:
                E, F = L["mlp"]["router"]["experts"], L["mlp"]["expert"]["ff"]
                t[f + "router"], t[f + "router.b"] = mat(E, D), around(E, 0.0, 0.5)
                for e in range(E):
                    t[f + f"e{e}.gate"], t[f + f"e{e}.up"], t[f + f"e{e}.down"] = mat(F, D), mat(F, D), mat(D, F)
        for n in names:
            t[f"l{i}.{n}"], t[f"l{i}.{n}.b"] = around(D, 1.0, 0.2), around(D, 0.0, 0.2)
    t["final.norm"], t["final.norm.b"] = around(D, 1.0, 0.2), around(D, 0.0, 0.2)
    t["head"] = mat(V, D, 3.0)
    return t


def stack(**kw):
    """Layers of different sizes and windows; latents read by later layers with narrower and wider windows."""
    return config([layer(), layer(heads=5, dim=16, rot_dim=12, vdim=8, q_rank=16, kv_rank=20, window=21, mlp=moe()),
                   layer(heads=2, dim=10, vdim=12, kv_from=0, window=17, scale=0.31, mlp=None),
                   layer(heads=4, rot_dim=12, kv_rank=20, q_rank=33, kv_from=1, window=4, mlp=moe(9, 3, 17)),
                   layer(window=6, base=50.0)], **kw)


def needle(window, sources=0, heads=2, seed=0, vocab=64, dim=16, vdim=16, rot_dim=8, kv_rank=24):
    """One mixer (or `sources` more that read its latents, with the same window) whose query for token 0 meets the key of
    token 1 with a score far above all others in the unrotated dimensions; values tell the tokens apart."""
    size = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=16, kv_rank=kv_rank, scale=1.0, mlp=None)
    layers = [layer(window=1 if sources else window, **size)] + [layer(window=window, kv_from=0, **size) for _ in range(sources)]
    cfg = config(layers, width=64, vocab=vocab, pairs=None, cap=30.0, alpha=1.0)
    t = tensors(cfg, seed)
    t["embed"] = 8.0 * np.eye(vocab, 64, dtype=np.float32)     # token = coordinate
    for i in range(len(layers)):
        p = f"l{i}.mix."
        last = i == len(layers) - 1
        t[p + "dq"][0] = 0.0
        t[p + "dq"][:, 0] = 0.0
        t[p + "dq"][0, 0] = 1.0                                # token 0 alone moves query latent 0
        u = t[p + "uq"].reshape(heads, dim + rot_dim, -1)
        u *= np.float32(0.125)
        u[:, :, 0] = 0.0
        u[:, 3] = 0.0
        u[:, 3, 0] = 4.0 if last else 0.0
        if i == 0:
            t[p + "dkv"][0] = 0.0
            t[p + "dkv"][:, 1] *= 0.25
            t[p + "dkv"][0, 1] = 1.0                           # token 1 alone moves latent 0
        k = t[p + "uk"].reshape(heads, dim, -1)
        k *= np.float32(0.125)
        k[:, :, 0] = 0.0
        k[:, 3] = 0.0
        k[:, 3, 0] = 1.0
        if not last:
            t[p + "o"] *= 0.0                                  # (the layers in front leave the tokens as they are)
            t[f"l{i}.norm1"], t[f"l{i}.norm1.b"] = np.ones(64, np.float32), np.zeros(64, np.float32)
    return cfg, t
