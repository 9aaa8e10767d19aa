"""Host side of the Rugesun model and the plain restatement it is tested against, without a GPU: config.json -> blocks,
tensors, and closed forms for the restatement's mechanisms."""
import numpy as np
import pytest

import rugesun_models as M
from nn_b200 import models, rugesun, safetensors
from nn_b200.decoder import ACT_GELU_TANH, MIXER_LATENT, MIXER_NONE
from oracle import rugesun_ref as ref


def test_blocks_from_config():
    cfg = M.stack(alpha=0.75)
    b = rugesun.layer_blocks(cfg)
    assert [(i, p) for i, p, _ in b] == [(0, "mix"), (0, "mlp"), (1, "mix"), (1, "mlp"), (2, "mix"), (3, "mix"), (3, "mlp"), (4, "mix"), (4, "mlp")]
    a, d, _, e, c, s = (x for _, _, x in b[:6])
    assert (a.mixer, a.heads, a.dim, a.rot_dims, a.vdim, a.q_rank, a.kv_rank, a.window, a.kv_from) == (MIXER_LATENT, 3, 24, 8, 20, 28, 36, 9, -1)
    assert (a.scale, a.rot_base, a.alpha, a.post_norm, a.ffn) == (0.23, 3e3, 0.75, True, 0)
    assert (d.mixer, d.ffn, d.ffn_act, d.experts, d.alpha) == (MIXER_NONE, 90, ACT_GELU_TANH, 0, 0.75)
    assert (e.mixer, e.ffn, e.experts, e.top, e.expert_ffn) == (MIXER_NONE, 0, 6, 2, 40)
    assert c.kv_from == 0 and s.kv_from == 2   # block numbers, not layer numbers


def test_configurations_that_cannot_be_right():
    for L in (dict(M.layer(), type="other"), M.layer(mlp={"kind": "routed", "ff": 8})):
        with pytest.raises(rugesun.ConfigError):
            rugesun.layer_blocks(M.config([L]))
    for layers in ([M.layer(kv_from=0)], [M.layer(), M.layer(kv_from=2), M.layer()], [M.layer(), M.layer(kv_from=0), M.layer(kv_from=1)]):
        with pytest.raises(rugesun.ConfigError):
            rugesun.layer_blocks(M.config(layers))
    L = M.layer()
    L["mixer"]["rot"]["dims"] = 4
    with pytest.raises(rugesun.ConfigError):
        rugesun.layer_blocks(M.config([L]))


def test_block_tensors_carry_every_tensor_of_the_model(tmp_path):
    cfg = M.stack()
    t = M.tensors(cfg)
    M.write_folder(tmp_path, cfg, t)
    f = safetensors.SafetensorsFile(str(tmp_path / "model.safetensors"))
    used = set()

    class Spy:
        def __init__(self, f):
            self.f = f

        def __getattr__(self, n):
            def get(name):
                used.add(name)
                return getattr(self.f, n)(name)
            return get

    for i, p, b in rugesun.layer_blocks(cfg):
        x = rugesun.block_tensors(Spy(f), i, p, b)
        for e in range(b.experts):
            gate, up, down = x.expert(e)
            assert np.array_equal(safetensors.bf16_to_f32(down), t[f"l{i}.mlp.e{e}.down"])
    assert used == {n for n in t if n.startswith("l")}


def test_registry():
    assert "Rugesun" in models.architectures()


# ---- closed forms for the restatement ----

def test_restated_pairs():
    assert ref.pair_rows([3, 5, 0, 5], 13, 4, 10) == [10, (39 + 20) % 10, 65 % 10, 20 % 10]


def test_restated_norm_and_activation():
    x = np.random.default_rng(0).standard_normal((4, 50)) * 3 + 2
    y = ref.layer_norm(x, np.full(50, 2.0), np.full(50, -1.0), 0.0)
    assert np.allclose(y.mean(-1), -1) and np.allclose(y.std(-1), 2)
    assert np.allclose(ref.layer_norm(np.zeros((1, 5)), np.ones(5), np.arange(5.0), 1e-5), np.arange(5.0))
    z = np.linspace(-4, 4, 17)
    from math import erf
    assert np.abs(ref.gelu_tanh(z) - [0.5 * v * (1 + erf(v / 2 ** 0.5)) for v in z]).max() < 1e-3 and abs(ref.gelu_tanh(1.0) - 0.841192) < 1e-6


def test_restated_route():
    idx, p = ref.route(np.array([[0.0, 3.0, 1.0, 2.0]]), 2)
    assert idx.tolist() == [[1, 3]] and np.allclose(p, [[1 / (1 + np.exp(-1)), 1 / (1 + np.e)]])


def test_restated_cap():
    assert np.allclose(ref.soft_cap(np.array([1e-6, 1e6]), 30.0), [1e-6, 30.0]) and ref.soft_cap(5.0, None) == 5.0


def test_restated_attention_is_the_absorbed_form():
    """Scores and values through the latent itself: q^T W_uk c = (W_uk^T q)^T c."""
    cfg = M.config([M.layer(mlp=None)])
    w = {n: t.astype(np.float64) for n, t in ref.part(M.tensors(cfg, 3), "l0.mix.").items()}
    m = cfg["layers"][0]["mixer"]
    x = np.random.default_rng(1).standard_normal((20, 72))
    kv = ref.latent(m, w, x, 1e-5)
    got = ref.latent_attention(m, w, x, kv, 1e-5, np.float64)
    (c, r), (qu, qr) = kv, ref.latent_queries(m, w, x, 1e-5)
    uk, uv = w["uk"].reshape(3, 24, 36), w["uv"].reshape(3, 20, 36)
    out = np.zeros((20, 3, 20))
    for h in range(3):
        s = (qu[:, h] @ uk[h] @ c.T + qr[:, h] @ r.T) * m["scale"]
        i, j = np.indices(s.shape)
        s[(j > i) | (i - j >= 9)] = -np.inf
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = p / p.sum(-1, keepdims=True) @ c @ uv[h].T
    assert np.allclose(got, out.reshape(20, -1) @ w["o"].T)


def test_needle_weights_make_one_score_stand_out():
    cfg, t = M.needle(5)
    ids = [3, 1, 7, 9, 4, 0, 8]
    far = ref.forward(cfg, t, [3, 6, 7, 9, 4, 0, 8])
    assert np.abs(ref.forward(cfg, t, ids)[5] - far[5]).max() > 0.1
