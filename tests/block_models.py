"""Small random models of the block decoder for the tests: config.json dicts, tensors (f32 values that are
exact in bf16) and folders on disk. Shares no code with the product."""
import json
import os
import struct

import numpy as np


def bf16_exact(x):
    u = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((u + ((u >> np.uint32(16)) & np.uint32(1)) + np.uint32(0x7FFF)) & np.uint32(0xFFFF0000)).view(np.float32)


def attention(heads=4, kv_heads=2, dim=24, vdim=20, window=9, conv=3, rot=(1e4, 16), scale=0.2, v_mix=True):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "scale": scale, "v_mix": v_mix,
         "rot": {"base": rot[0], "dims": rot[1]}}
    if conv:
        m["conv"] = conv
    return {"type": "attention", "mixer": m}


def gla(heads=3, dim=20, vdim=28, tau=4.0, rank=6):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "_rank": rank}


def retention(heads=3, dim=24, vdim=12, decay=(0.6, 0.9, 0.98), rot=(1e3, 24)):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), "rot": {"base": rot[0], "dims": rot[1]}}}


def config(layers, width=72, vocab=150, ff=90, eps=1e-5):
    out = []
    for L in layers:
        L = dict(L)
        L.setdefault("mlp", {"kind": "dense", "ff": ff})
        out.append(L)
    return {"architecture": "Sikivik", "layers": out, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def tensors(cfg, seed=0):
    rng = np.random.default_rng(seed)
    D, V = cfg["width"], cfg["vocab"]

    def mat(n, k, gain=1.0):
        return bf16_exact(rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def around(n, mean, spread):
        return bf16_exact(mean + spread * rng.standard_normal(n))

    t = {"embed": bf16_exact(rng.standard_normal((V, D)))}
    for i, L in enumerate(cfg["layers"]):
        m, p = L["mixer"], f"l{i}.mix."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        t[f"l{i}.norm1"] = around(D, 1.0, 0.2)
        G = m.get("kv_heads", H)
        widths = {"q": H * d, "k": G * d, "v": G * e}
        for n, w in widths.items():
            t[p + n] = mat(w, D, 1.5)
        t[p + "g"], t[p + "o"] = mat(H * e, D), mat(D, H * e)
        if L["type"] == "attention":
            for n, w in widths.items():
                t[p + n + ".b"] = around(w, 0.0, 0.3)
                if m.get("conv"):
                    t[p + n + ".conv"] = bf16_exact(rng.standard_normal((w, m["conv"])) * 0.7)
            t[p + "o.b"] = around(D, 0.0, 0.2)
            if m.get("v_mix"):
                t[p + "vmix"] = bf16_exact(np.float32(0.3 + 0.1 * i)).reshape(())
        elif L["type"] == "gla":
            r = L["_rank"]
            t[p + "a1"], t[p + "a2"], t[p + "a2.b"] = mat(r, D), mat(H * d, r), around(H * d, 1.0, 1.0)
            t[p + "norm"] = around(e, 1.0, 0.3)
        if L.get("mlp"):
            F = L["mlp"]["ff"]
            q = f"l{i}.mlp."
            t[q + "gate"], t[q + "up"], t[q + "down"] = mat(F, D), mat(F, D), mat(D, F)
    t["final.norm"] = around(D, 1.0, 0.2)
    t["head"] = mat(V, D)
    return t


def write_folder(folder, cfg, t):
    clean = dict(cfg, layers=[{k: v for k, v in L.items() if not k.startswith("_")} for L in cfg["layers"]])
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(clean, f)
    head, at, blobs = {}, 0, []
    for name, a in t.items():
        b = (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[name] = {"dtype": "BF16", "shape": list(np.shape(a)), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    js = json.dumps(head).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(js)) + js + b"".join(blobs))
    return folder
