"""Block decoders on the device against the plain restatement (oracle/hybrid_ref.py): every mixer alone, the
whole stack, prompts cut into portions, decoding through the caches and states, greedy generation, the
command lines. Models are small, random and made here; where random weights would hide a fault the weights
are made so that one score stands out."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

torch = pytest.importorskip("torch")

import block_models as M
from nn_b200 import api, models
from nn_b200.decoder import BlockConfig, BlockDecoder
from oracle import hybrid_ref as ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 2e-5, 4e-2   # root mean square of the difference over that of the expected logits


def load(tmp_path, cfg, t, dtype=api.F32, max_seq=256, block_rows=0):
    folder = tmp_path / "model"
    folder.mkdir(exist_ok=True)
    M.write_folder(folder, cfg, t)
    return models.load_model(str(folder), max_seq=max_seq, act_dtype=dtype, block_rows=block_rows)


def err(got, want):
    d = np.asarray(got, np.float64) - want
    return float(np.sqrt((d * d).mean(-1)).max() / np.sqrt((want * want).mean()))


def run(dec, tokens, cuts):
    """All logits of a sequence fed in portions of the given sizes (the rest in one)."""
    out, at = [], 0
    for n in list(cuts) + [len(tokens)]:
        part = tokens[at:at + n]
        if not part:
            break
        out.append(dec.extend(part, at, list(range(len(part)))))
        at += len(part)
    return np.concatenate(out)


def tokens(n, vocab, seed=1):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


MIXERS = {
    "attention": [M.attention()],
    "attention, no feed-forward": [dict(M.attention(), mlp=None)],
    "no convolution": [M.attention(conv=0)],
    "one tap": [M.attention(conv=1)],
    "two taps": [M.attention(conv=2, window=4)],
    "five taps": [M.attention(conv=5)],
    "window of one": [M.attention(window=1)],
    "window past the sequence": [M.attention(window=500)],
    "one key head, odd sizes": [M.attention(heads=6, kv_heads=1, dim=10, vdim=7, rot=(5e4, 6))],
    "a key head per query head": [M.attention(heads=5, kv_heads=5, dim=16, vdim=16, rot=(100.0, 16))],
    "twelve query heads per key head": [M.attention(heads=24, kv_heads=2, dim=8, vdim=8, rot=(1e4, 4))],
    "wide heads": [M.attention(heads=2, kv_heads=1, dim=132, vdim=200, rot=(1e4, 128), scale=0.05)],
    "value mixing over three layers": [M.attention(), M.attention(v_mix=False), M.attention(window=5), M.attention(heads=8, kv_heads=2, dim=8, rot=(10.0, 8))],
    "gla": [M.gla()],
    "gla, rank one": [M.gla(rank=1, tau=1.0)],
    "gla, value heads wider than a tile": [M.gla(heads=2, dim=33, vdim=50, rank=19)],
    "gla, large heads": [dict(M.gla(heads=1, dim=256, vdim=160), mlp=None)],
    "gla, five key groups": [M.gla(heads=1, dim=150, vdim=40)],
    "retention": [M.retention()],
    "retention, part of the head rotated": [M.retention(heads=2, dim=70, vdim=33, decay=(0.5, 0.999), rot=(50.0, 10))],
    "retention, large heads": [M.retention(heads=1, dim=200, vdim=96, decay=(0.97,), rot=(1e4, 200))],
}


@pytest.mark.parametrize("name", sorted(MIXERS))
def test_each_mixer_in_prompts_and_decoding(tmp_path, name):
    cfg = M.config(MIXERS[name])
    t = M.tensors(cfg, seed=len(name))
    ids = tokens(45, cfg["vocab"])
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t)
    assert err(run(dec, ids, []), want) <= F32_TOL
    assert err(run(dec, ids, [1] * 45), want) <= F32_TOL
    assert err(run(dec, ids, [17, 2, 3, 1, 9]), want) <= F32_TOL
    dec.release()
    dec = load(tmp_path, cfg, t, api.BF16)
    assert err(run(dec, ids, []), want) <= BF16_TOL
    assert err(run(dec, ids, [20] + [1] * 25), want) <= BF16_TOL
    dec.release()


def stack(**kw):
    return M.config([M.attention(), M.gla(), M.retention(), M.gla(heads=2, dim=8, vdim=8, rank=3), M.attention(window=14), M.retention()], **kw)


@pytest.mark.parametrize("width,ff,vocab", [(72, 90, 150), (64, 64, 128), (100, 33, 77), (136, 256, 641), (7, 5, 11)])
def test_whole_stack_at_several_widths(tmp_path, width, ff, vocab):
    cfg = stack(width=width, ff=ff, vocab=vocab)
    t = M.tensors(cfg, seed=width)
    ids = tokens(40, vocab)
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t)
    assert err(run(dec, ids, [30] + [1] * 10), want) <= F32_TOL
    dec.release()
    dec = load(tmp_path, cfg, t, api.BF16)
    assert err(run(dec, ids, [30] + [1] * 10), want) <= BF16_TOL
    dec.release()


@pytest.mark.parametrize("depth", [1, 2, 3, 5])
def test_layer_by_layer(tmp_path, depth):
    cfg = stack()
    cfg["layers"] = cfg["layers"][:depth]
    t = M.tensors(cfg, seed=3)
    ids = tokens(25, cfg["vocab"])
    dec = load(tmp_path, cfg, t)
    assert err(run(dec, ids, []), ref.forward(cfg, t, ids)) <= F32_TOL
    dec.release()


@pytest.mark.parametrize("cuts", [[2] * 60, [3] * 40, [5, 1, 1, 7, 2] * 8, [8] * 15, [64, 2], [119], [1, 119]], ids=str)
@pytest.mark.parametrize("rows", [0, 16])
def test_portions_do_not_change_the_logits(tmp_path, cuts, rows):
    """Also with row blocks of 16, so that a portion is cut again inside and the key ring wraps."""
    cfg = stack()
    t = M.tensors(cfg, seed=5)
    ids = tokens(120, cfg["vocab"])
    dec = load(tmp_path, cfg, t, block_rows=rows)
    assert err(run(dec, ids, cuts), ref.forward(cfg, t, ids)) <= F32_TOL
    dec.release()


def test_portions_on_the_tensor_core_products(tmp_path):
    """bf16: 300 rows take the large-batch product, 5 .. 255 the middle one, 1 .. 4 the row kernel."""
    cfg = stack(width=128, ff=192, vocab=200)
    t = M.tensors(cfg, seed=6)
    ids = tokens(310, cfg["vocab"])
    want = ref.forward(cfg, t, ids, np.float32)
    dec = load(tmp_path, cfg, t, api.BF16, max_seq=400)
    for cuts in ([300], [128, 64, 100, 5, 4, 2, 1], [290] + [1] * 20):
        assert err(run(dec, ids, cuts), want) <= BF16_TOL
    dec.release()


def test_a_restart_finds_nothing_of_the_sequence_before(tmp_path):
    cfg = stack()
    t = M.tensors(cfg, seed=7)
    a, b = tokens(50, cfg["vocab"], 1), tokens(33, cfg["vocab"], 2)
    for dtype in (api.F32, api.BF16):
        dec = load(tmp_path, cfg, t, dtype)
        fresh = run(dec, b, [20, 1, 1])
        run(dec, a, [40] + [1] * 10)
        assert np.array_equal(run(dec, b, [20, 1, 1]), fresh)
        run(dec, a, [2])
        run(dec, [5], [])
        assert np.array_equal(run(dec, b, [20, 1, 1]), fresh)
        first = run(dec, b[:1], [])
        assert err(first, ref.forward(cfg, t, b[:1])) <= (F32_TOL if dtype == api.F32 else BF16_TOL)
        dec.release()


def test_logits_of_some_positions_only(tmp_path):
    cfg = stack()
    t = M.tensors(cfg, seed=8)
    ids = tokens(100, cfg["vocab"])
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t, block_rows=32)
    assert dec.extend(ids[:10], 0).shape == (0, cfg["vocab"])
    pick = [0, 21, 22, 53, 54, 89]
    assert err(dec.extend(ids[10:], 10, pick), want[[10 + p for p in pick]]) <= F32_TOL
    everything = dec.extend(ids, 0, list(range(100)))   # more rows than are formed together
    assert err(everything, want) <= F32_TOL
    with pytest.raises(api.InvalidArgument):
        dec.extend(ids[:4], 0, [2, 1])
    with pytest.raises(api.InvalidArgument):
        dec.extend(ids[:4], 0, [4])
    dec.release()


# ---- windows: one key stands out, and the answer depends on whether it is seen ----

def needle_model(window, vocab=64, heads=2, kv_heads=1, taps=2, seed=0):
    """One attention layer whose query for token 0 meets the key of token 1 with a score far above all others
    (in the dimensions that are not rotated), and whose values tell the tokens apart."""
    L = dict(M.attention(heads=heads, kv_heads=kv_heads, dim=16, vdim=16, window=window, conv=taps, rot=(1e4, 8), scale=1.0, v_mix=False), mlp=None)
    cfg = M.config([L], width=64, vocab=vocab)
    t = M.tensors(cfg, seed)
    t["embed"] = np.eye(vocab, 64, dtype=np.float32)          # token = coordinate
    p = "l0.mix."
    t["l0.norm1"] = np.full(64, 0.125, np.float32)            # one-hot rows of width 64: h = one-hot
    for n in "qk":
        t[p + n] *= 0.125
        t[p + n + ".b"] *= 0.125
        w = t[p + n].reshape(-1, 16, 64)
        w[:, 8:, :] = 0.0
        w[:, 12, 0 if n == "q" else 1] = 5.0
        c = np.zeros_like(t[p + n + ".conv"])
        c[:, -1] = 1.0
        t[p + n + ".conv"] = c
    c = np.zeros_like(t[p + "v.conv"])
    c[:, -1] = 1.0
    t[p + "v.conv"] = c
    return cfg, t


@pytest.mark.parametrize("window", [2, 5, 32, 33, 64, 97])
def test_key_just_inside_and_just_outside_the_window(tmp_path, window):
    cfg, t = needle_model(window)
    rng = np.random.default_rng(window)
    dec = load(tmp_path, cfg, t, max_seq=512, block_rows=24)
    for start in (0, 1, 40):   # where the key lies: the first token, the second, further on
        seen = []
        for distance in (window - 1, window):
            ids = rng.integers(2, 64, start + distance + 4).tolist()
            ids[start] = 1
            ids[start + distance] = 0
            want = ref.forward(cfg, t, ids)
            q = start + distance
            for cuts in ([], [q] + [1] * 4, [max(1, q - 1), 2], [start + 1], [7] * 40):
                assert err(run(dec, ids, cuts), want) <= F32_TOL
            other = list(ids)
            other[start] = 2
            seen.append(err(ref.forward(cfg, t, other)[q:q + 1], want[q:q + 1]))
        assert seen[0] > 0.1 and seen[1] < 1e-9   # inside it decides the answer, outside it is gone
    dec.release()


@pytest.mark.parametrize("dtype,tol", [(api.F32, F32_TOL), (api.BF16, BF16_TOL)])
def test_long_decoding_over_a_ring_that_wraps(tmp_path, dtype, tol):
    """Several hundred decoded tokens; the key ring holds window - 1 + 8 positions and wraps many times. The
    needle is met at the window's edges all along."""
    window = 37
    cfg, t = needle_model(window, heads=3, kv_heads=3)
    ids = np.random.default_rng(4).integers(2, 64, 420).tolist()
    for p in range(5, 380, 29):
        ids[p] = 1
        ids[p + window - 1 + (p % 2)] = 0
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t, dtype, max_seq=512, block_rows=8)
    assert err(run(dec, ids, [11] + [1] * 409), want) <= tol
    dec.release()


def test_long_window_over_several_decode_ranges(tmp_path):
    """A window of 300 keys is dealt to three groups of warps whose partial sums are merged."""
    cfg, t = needle_model(300, heads=4, kv_heads=2)
    ids = np.random.default_rng(9).integers(2, 64, 340).tolist()
    ids[3], ids[302], ids[38], ids[337], ids[339] = 1, 0, 1, 0, 0
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t, max_seq=400)
    assert err(run(dec, ids, [295] + [1] * 45), want) <= F32_TOL
    assert err(run(dec, ids, []), want) <= F32_TOL
    dec.release()


def test_a_far_token_is_held_by_the_recurrent_state(tmp_path):
    """Decays close to one: the first token still moves the last logits, and it does so by the right amount."""
    for L in (M.retention(heads=2, dim=16, vdim=16, decay=(0.9999, 0.995), rot=(1e4, 8)), M.gla(heads=2, dim=16, vdim=16, tau=200.0)):
        cfg = M.config([dict(L, mlp=None)], width=64, vocab=64)
        t = M.tensors(cfg, 11)
        ids = tokens(150, 64, 3)
        want = ref.forward(cfg, t, ids)
        changed = ref.forward(cfg, t, [(ids[0] + 1) % 64] + ids[1:])
        assert err(changed[-1:], want[-1:]) > 1e-3
        dec = load(tmp_path, cfg, t)
        for cuts in ([], [1] + [2] * 20, [100] + [1] * 50):
            assert err(run(dec, ids, cuts), want) <= F32_TOL
        dec.release()


# ---- generation, sequence keeping, command lines ----

def greedy(cfg, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(ref.forward(cfg, t, ids, np.float32)[-1].argmax()))
    return ids[len(prompt):]


def test_greedy_generation(tmp_path):
    cfg = stack()
    t = M.tensors(cfg, seed=13)
    prompt = tokens(23, cfg["vocab"])
    want = greedy(cfg, t, prompt, 24)
    dec = load(tmp_path, cfg, t)
    assert dec.complete(prompt, 24) == want
    assert dec.complete(prompt, 24, use_graph=False) == want
    # after the replayed graphs the decoder knows where it is: the sequence goes on from there
    assert dec.state()[1] == len(prompt) + 23
    more = dec.extend(want[-1:], len(prompt) + 23, [0])
    assert int(more[0].argmax()) == greedy(cfg, t, prompt, 25)[-1]
    dec.release()


def test_a_sequence_continues_only_where_its_state_is(tmp_path):
    cfg = stack()
    dec = load(tmp_path, cfg, M.tensors(cfg, seed=1), max_seq=32)
    dec.extend([1, 2, 3], 0)
    for pos in (1, 2, 4):
        with pytest.raises(api.InvalidArgument):
            dec.extend([4], pos)
        with pytest.raises(api.InvalidArgument):
            dec.extend([4, 5], pos)
    dec.extend([4, 5], 3)
    with pytest.raises(api.Unsupported):
        dec.extend([1] * 28, 5)
    dec.extend([1] * 27, 5)
    with pytest.raises(api.Unsupported):
        dec.step()
    dec.extend([1], 0)
    dec.release()


def test_shapes_are_checked():
    b = api.gpu_backend()
    for bad in (dict(heads=3, kv_heads=2), dict(rot_dims=5), dict(dim=8, rot_dims=10), dict(heads=0), dict(vdim=300)):
        with pytest.raises(api.TensorError):
            BlockDecoder(b, hidden=64, vocab=10, blocks=[BlockConfig(**bad)], max_seq=8)
    with pytest.raises(api.TensorError):
        BlockDecoder(b, hidden=64, vocab=10, blocks=[BlockConfig(mixer=1, dim=300)], max_seq=8)


def test_trace_and_generation_command_lines(tmp_path):
    cfg = stack()
    t = M.tensors(cfg, seed=17)
    folder = tmp_path / "m"
    folder.mkdir()
    M.write_folder(folder, cfg, t)
    out = tmp_path / "out"
    out.mkdir()
    a, b = tokens(30, cfg["vocab"], 5), tokens(9, cfg["vocab"], 6)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [19, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:21], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": a[21:], "want": [0, 8]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": b, "want": [8]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    wa, wb = ref.forward(cfg, t, a), ref.forward(cfg, t, b)
    for step, want in ((0, wa[[19, 3]]), (2, wa[[21, 29]]), (3, wb[[8]])):
        assert err(np.fromfile(out / f"{step}.f32", "<f4").reshape(want.shape), want) <= F32_TOL
    assert not (out / "1.f32").exists()
    r = subprocess.run([sys.executable, "-m", "nn_b200.generate", "--model", str(folder), "--prompt", ",".join(map(str, b)), "--new", "6",
                        "--dtype", "float32"], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr
    assert r.stdout.strip() == ",".join(map(str, greedy(cfg, t, b, 6)))


# ---- the f32 product path ----

@pytest.mark.parametrize("m,n,k", [(1, 70, 64), (5, 64, 96), (9, 130, 320), (200, 65, 1024)])
@pytest.mark.parametrize("fmt", ["bf16", "f32"])
def test_f32_products_round_nothing(m, n, k, fmt):
    from nn_b200.formats import QuantFormat as Q
    rng = np.random.default_rng(m)
    w = M.bf16_exact(rng.standard_normal((n, k))) if fmt == "bf16" else rng.standard_normal((n, k)).astype(np.float32)
    x = rng.standard_normal((m, k)).astype(np.float32)
    raw = (w.view(np.uint32) >> 16).astype(np.uint16).view(np.uint8) if fmt == "bf16" else w.view(np.uint8)
    t = api.from_quantized(raw, Q.BF16_DENSE if fmt == "bf16" else Q.F32_DENSE, [n, k])
    t.backend.set_path(api.PATH_F32)
    try:
        y = api.quantized_linear(torch.from_numpy(x).to("cuda:0"), t, None, out_dtype=torch.float32).cpu().numpy()
    finally:
        t.backend.set_path(api.PATH_AUTO)
    want = x.astype(np.float64) @ w.astype(np.float64).T
    assert np.abs(y - want).max() <= 2e-6 * np.sqrt(k) * np.abs(want).max()
    t.release()


@pytest.mark.parametrize("n,k", [(1, 64), (7, 128), (300, 256), (1000, 1536), (333, 5056), (4096, 4096), (50, 40000), (70000, 512)])
@pytest.mark.parametrize("m", [1, 2, 3, 4])
def test_row_product_of_bf16_weights(n, k, m):
    """One to four rows: the streaming kernel multiplies bf16 by bf16 exactly and sums in f32."""
    from nn_b200.formats import QuantFormat as Q
    b = api.gpu_backend()
    gen = torch.Generator(device="cuda:0")
    gen.manual_seed(n + k)
    w = torch.randn(n, k, device="cuda:0", generator=gen).to(torch.bfloat16)
    x = torch.randn(m, k, device="cuda:0", generator=gen).to(torch.bfloat16)
    bias = torch.randn(n, device="cuda:0", generator=gen)
    t = api.DeviceWeight.from_device(b, Q.BF16_DENSE, w.view(torch.uint8).reshape(-1), n, k)
    y = torch.full((m, n), float("nan"), device="cuda:0")
    b.check(b._lib.nnq_linear(b._ctx, t.handle(), x.data_ptr(), api.BF16, m, bias.data_ptr(), y.data_ptr(), api.F32, api._stream_ptr(None)))
    want = x.double() @ w.double().T + bias.double()
    assert float((y.double() - want).abs().max() / want.abs().max()) <= 1e-5
    b.device_status()
    t.release()


# ---- attention of a block of rows on the tensor cores (bf16 decoders) ----

@pytest.mark.parametrize("heads,kv,dim,vdim,window", [(4, 2, 24, 20, 9), (8, 1, 88, 56, 100), (6, 3, 128, 128, 70), (4, 4, 64, 40, 300), (12, 2, 72, 100, 33),
                                                       (5, 5, 8, 8, 1), (16, 2, 128, 96, 2000)])
def test_tensor_core_attention_is_as_exact_as_the_decode_kernel(tmp_path, heads, kv, dim, vdim, window):
    """A bf16 decoder's prompt pass (operands split into two bf16 terms) against its own decode steps (f32 on the
    CUDA cores): everything before and after the attention rounds alike, so the two agree far more closely than
    either agrees with the unrounded model."""
    cfg = M.config([M.attention(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, window=window, rot=(1e4, dim // 4 * 2), scale=3.0 * dim ** -0.5)], width=64, vocab=96)
    t = M.tensors(cfg, seed=heads)
    ids = tokens(330, 96, 2)
    dec = load(tmp_path, cfg, t, api.BF16, max_seq=400, block_rows=150)
    want = run(dec, ids, [1] * 330).astype(np.float64)
    for cuts in ([], [40, 111, 33], [200]):
        d = run(dec, ids, cuts) - want
        assert np.sqrt((d * d).mean() / (want * want).mean()) <= 2e-3, cuts
    assert err(want, ref.forward(cfg, t, ids, np.float32)) <= BF16_TOL
    dec.backend.device_status()
    dec.release()
