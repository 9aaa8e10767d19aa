"""Host side of the block decoder and the plain restatement it is tested against, without a GPU: the
safetensors container, config.json -> block configurations, the registry, the trace replay's sequence keeping,
and closed forms for the restatement's mechanisms."""
import json

import numpy as np
import pytest

import block_models as M
from nn_b200 import models, safetensors, sikivik, trace
from nn_b200.decoder import MIXER_ATTENTION, MIXER_RECURRENT
from oracle import hybrid_ref as ref


def test_safetensors_round_trip(tmp_path):
    p = str(tmp_path / "t.safetensors")
    x = np.array([[1.0, -2.5, 3.0e-8], [7.0, 0.0, -1e30]], np.float32)
    bits = safetensors.f32_to_bf16(x)
    safetensors.write_safetensors(p, {"a": ("BF16", (2, 3), bits), "s": ("BF16", (), bits[0, 1]), "b": ("F32", (2, 3), x),
                                      "i": ("I32", (2,), np.array([3, -4]))})
    f = safetensors.SafetensorsFile(p)
    assert np.array_equal(f.f32("a"), M.bf16_exact(x)) and np.array_equal(f.bf16("a"), bits)
    assert np.array_equal(f.bf16("b"), bits) and np.array_equal(f.f32("b"), x)
    assert f.f32("s").shape == () and float(f.f32("s")) == -2.5
    assert f.raw("i").tolist() == [3, -4] and f.info("i").shape == (2,)
    with pytest.raises(safetensors.SafetensorsError):
        f.info("missing")


def test_safetensors_refuses_ranges_that_do_not_fit(tmp_path):
    for head in ({"a": {"dtype": "F32", "shape": [4], "data_offsets": [0, 12]}}, {"a": {"dtype": "F32", "shape": [4], "data_offsets": [0, 16]}},
                 {"a": {"dtype": "Q9", "shape": [1], "data_offsets": [0, 4]}}):
        p = tmp_path / "bad.safetensors"
        js = json.dumps(head).encode()
        p.write_bytes(len(js).to_bytes(8, "little") + js + b"\0" * 8)
        with pytest.raises(safetensors.SafetensorsError):
            safetensors.SafetensorsFile(str(p))


def test_block_configurations_from_config():
    cfg = M.config([M.attention(conv=0), M.attention(window=40), dict(M.gla(), mlp=None), M.retention()], ff=55)
    a, a2, g, r = (sikivik.block_config(L, 6 if L["type"] == "gla" else 0) for L in cfg["layers"])
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.conv_taps, a.ffn) == (MIXER_ATTENTION, 4, 2, 24, 20, 9, 0, 55)
    assert (a.rot_dims, a.rot_base, a.scale, a.value_mix, a.out_gate) == (16, 1e4, 0.2, True, True)
    assert (a2.window, a2.conv_taps) == (40, 3)
    assert (g.mixer, g.ffn, g.decay_rank, g.decay_tau, g.k_scale, g.rot_dims) == (MIXER_RECURRENT, 0, 6, 4.0, 1.0, 0)
    assert g.q_scale == 20 ** -0.5
    assert (r.mixer, r.decay_rank, r.q_scale, r.rot_dims, r.rot_base) == (MIXER_RECURRENT, 0, 1.0, 24, 1e3) and r.k_scale == 24 ** -0.5
    with pytest.raises(sikivik.ConfigError):
        sikivik.block_config({"type": "other", "mixer": dict(M.gla()["mixer"]), "mlp": None})
    with pytest.raises(sikivik.ConfigError):
        sikivik.block_config(dict(M.retention(decay=(0.5,)), mlp=None))
    with pytest.raises(sikivik.ConfigError):
        sikivik.block_config(dict(M.gla(), mlp={"kind": "routed", "ff": 8}))


def test_block_tensors_carry_every_tensor_of_the_model(tmp_path):
    cfg = M.config([M.attention(), M.gla(), M.retention()])
    t = M.tensors(cfg)
    M.write_folder(tmp_path, cfg, t)
    f = safetensors.SafetensorsFile(str(tmp_path / "model.safetensors"))
    b = [sikivik.block_tensors(f, i, L) for i, L in enumerate(cfg["layers"])]
    assert np.array_equal(safetensors.bf16_to_f32(b[0].q), t["l0.mix.q"]) and np.array_equal(b[0].v_bias, t["l0.mix.v.b"])
    assert np.array_equal(b[0].conv, np.concatenate([t[f"l0.mix.{n}.conv"] for n in "qkv"]))
    assert b[0].value_lambda == float(t["l0.mix.vmix"])
    assert np.array_equal(b[1].decay_w, t["l1.mix.a2"]) and np.array_equal(b[1].head_norm, t["l1.mix.norm"]) and b[1].decay is None
    assert np.allclose(b[2].decay, [0.6, 0.9, 0.98]) and b[2].head_norm is None and b[2].q_bias is None
    assert np.array_equal(safetensors.bf16_to_f32(b[2].down), t["l2.mlp.down"])


def test_registry(tmp_path):
    assert "Sikivik" in models.architectures() and "qwen3" in models.architectures()
    (tmp_path / "config.json").write_text('{"architecture": "Nobody"}')
    with pytest.raises(models.UnknownArchitecture):
        models.load_model(str(tmp_path), max_seq=8)


class FakeDecoder:
    def __init__(self):
        self.calls = []

    def extend(self, tokens, pos, want, stream):
        self.calls.append((list(tokens), pos, list(want)))
        return np.array([[float(w), float(pos)] for w in want], np.float32).reshape(len(want), 2)


def test_replay_keeps_one_sequence():
    d = FakeDecoder()
    r = trace.Replay(d, stream=0)
    assert r.step([{"id": "a", "tokens": [1, 2, 3], "want": []}]) is None
    got = r.step([{"id": "a", "tokens": [4, 5, 6], "want": [2, 0, 2]}], ["a"])
    assert got[:, 0].tolist() == [2.0, 0.0, 2.0] and got[0, 1] == 3.0
    r.step([{"id": "b", "tokens": [7], "want": [0]}])
    assert d.calls == [([1, 2, 3], 0, []), ([4, 5, 6], 3, [0, 2]), ([7], 0, [0])]
    with pytest.raises(ValueError):
        r.step([{"id": "c", "tokens": [1], "want": []}])
    with pytest.raises(ValueError):
        r.step([{"id": "b", "tokens": [1], "want": []}, {"id": "c", "tokens": [1], "want": []}])
    r.step([], ["b"])
    r.step([{"id": "c", "tokens": [1], "want": []}])
    assert d.calls[-1] == ([1], 0, [])


# ---- closed forms for the restatement ----

def test_restated_convolution():
    u = np.arange(1.0, 7.0).reshape(3, 2)
    assert np.allclose(ref.causal_conv(u, np.array([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]])), [[1, 0], [3, 0], [5, 2]])


def test_restated_rotation_is_relative():
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((2, 1, 1, 8))
    dot = lambda a, b: float((ref.rotate_half(q, 100.0, 6, np.array([a])) * ref.rotate_half(k, 100.0, 6, np.array([b]))).sum())
    assert abs(dot(3.0, 1.0) - dot(13.0, 11.0)) < 1e-12 and abs(dot(3.0, 1.0) - dot(3.0, 2.0)) > 1e-3
    assert np.array_equal(ref.rotate_half(q, 100.0, 6, np.array([5.0]))[..., 6:], q[..., 6:])


def test_restated_window():
    T = 7
    v = np.eye(T)[:, None, :]
    q = k = np.zeros((T, 1, 4))
    o = ref.window_attention(q, k, v, 1.0, 3)[:, 0]
    assert np.allclose(o[0], np.eye(T)[0]) and np.allclose(o[5], [0, 0, 0, 1 / 3, 1 / 3, 1 / 3, 0])
    assert np.allclose(ref.window_attention(q, k, v, 1.0, None)[6, 0], 1 / 7)


def test_restated_recurrence():
    rng = np.random.default_rng(1)
    q, k, a = rng.standard_normal((3, 5, 1, 4))
    a = ref.sigmoid(a)
    v = rng.standard_normal((5, 1, 3))
    o, _ = ref.decayed_state(q, k, v, a)
    for t in range(5):
        w = [np.sum(q[t, 0] * k[s, 0] * np.prod(a[s + 1:t + 1, 0], axis=0)) for s in range(t + 1)]
        assert np.allclose(o[t, 0], sum(x * v[s, 0] for s, x in enumerate(w)))
    z = np.array([[0.3, -2.0]])
    eye = np.eye(2)
    assert np.allclose(ref.gla_decay(z, eye, eye, np.zeros(2), 4.0), ref.sigmoid(z) ** 0.25)
