"""The Rugesun decoder on the device against the plain restatement (oracle/rugesun_ref.py): every mechanism alone, the
whole stack, prompts cut into portions, decoding through the latent rings, windows at their edges, greedy generation,
the command lines. Models are small, random and made here; where random weights would hide a fault the weights are made
so that one score stands out."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

torch = pytest.importorskip("torch")

import rugesun_models as M
from nn_b200 import api, models
from nn_b200.decoder import BlockConfig, BlockDecoder, MIXER_LATENT, MIXER_NONE
from oracle import rugesun_ref as ref

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL, BF16_TOL = 2e-5, 4e-2   # root mean square of the difference over that of the expected logits


def load(tmp_path, cfg, t, dtype=api.F32, max_seq=256, block_rows=0):
    folder = tmp_path / "model"
    folder.mkdir(exist_ok=True)
    M.write_folder(folder, cfg, t)
    return models.load_model(str(folder), max_seq=max_seq, act_dtype=dtype, block_rows=block_rows)


def errs(got, want):
    d = np.asarray(got, np.float64) - want
    return np.sqrt((d * d).mean(-1)) / np.sqrt((want * want).mean())


def err(got, want):
    return float(errs(got, want).max())


def close_bf16(got, want, tol=BF16_TOL):
    """Nine positions of ten within the tolerance: a rounded router input may choose another expert at a close call."""
    return float(np.quantile(errs(got, want), 0.9)) <= tol


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


MECHANISMS = {
    "latent attention alone": ([M.layer(mlp=None)], {}),
    "no pairs, no cap": ([M.layer(mlp=None)], dict(pairs=None, cap=None)),
    "pairs with large factors": ([M.layer(mlp=None)], dict(pairs=(7, 1000003, 2000000011))),
    "one bucket": ([M.layer(mlp=None)], dict(pairs=(1, 3, 4))),
    "a tight cap": ([M.layer(mlp=None)], dict(cap=0.8)),
    "alpha of one half": ([M.layer(), M.layer(mlp=M.moe())], dict(alpha=0.5)),
    "large eps": ([M.layer(), M.layer(mlp=M.moe())], dict(eps=0.3)),
    "window of one": ([M.layer(window=1)], {}),
    "window past the sequence": ([M.layer(window=500)], {}),
    "one head": ([M.layer(heads=1, dim=6, rot_dim=2, vdim=5, q_rank=4, kv_rank=3)], {}),
    "nine heads": ([M.layer(heads=9, dim=8, rot_dim=8, vdim=8)], {}),
    "no rotated part": ([M.layer(rot_dim=0)], {}),
    "more rotated than not": ([M.layer(dim=8, rot_dim=72, vdim=70, kv_rank=65, q_rank=130)], {}),
    "wide heads": ([M.layer(heads=2, dim=130, rot_dim=64, vdim=200, kv_rank=200, q_rank=70, scale=0.05)], {}),
    "heads of the tensor cores' sizes": ([M.layer(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=256, q_rank=192, scale=0.07)], {}),
    "a latent above 512": ([M.layer(heads=2, kv_rank=600, rot_dim=16)], {}),
    "dense feed-forward of odd width": ([M.layer(mlp={"kind": "dense", "ff": 33})], {}),
    "experts": ([M.layer(mlp=M.moe())], {}),
    "one expert of one": ([M.layer(mlp=M.moe(1, 1, 8))], {}),
    "every expert": ([M.layer(mlp=M.moe(5, 5, 12))], {}),
    "many experts": ([M.layer(mlp=M.moe(70, 8, 6))], {}),
    "latents of an earlier layer": ([M.layer(), M.layer(kv_from=0, heads=5, dim=12, vdim=9, q_rank=11)], {}),
    "latents read with a wider window": ([M.layer(window=3), M.layer(kv_from=0, window=30), M.layer(kv_from=0, window=12)], {}),
}


@pytest.mark.parametrize("name", sorted(MECHANISMS))
def test_each_mechanism_in_prompts_and_decoding(tmp_path, name):
    layers, kw = MECHANISMS[name]
    cfg = M.config(layers, **kw)
    t = M.tensors(cfg, seed=len(name))
    ids = tokens(45, cfg["vocab"])
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t)
    assert err(run(dec, ids, []), want) <= F32_TOL
    assert err(run(dec, ids, [1] * 45), want) <= F32_TOL
    assert err(run(dec, ids, [17, 2, 3, 1, 9]), want) <= F32_TOL
    dec.release()
    dec = load(tmp_path, cfg, t, api.BF16)
    assert close_bf16(run(dec, ids, []), want)
    assert close_bf16(run(dec, ids, [20] + [1] * 25), want)
    assert close_bf16(run(dec, ids, [2] * 10 + [8, 1, 13]), want)
    dec.backend.device_status()
    dec.release()


@pytest.mark.parametrize("width,vocab", [(72, 150), (64, 128), (101, 77), (136, 641), (7, 11)])
def test_whole_stack_at_several_widths(tmp_path, width, vocab):
    cfg = M.stack(width=width, vocab=vocab)
    t = M.tensors(cfg, seed=width)
    ids = tokens(40, vocab)
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t)
    assert err(run(dec, ids, [30] + [1] * 10), want) <= F32_TOL
    dec.release()
    dec = load(tmp_path, cfg, t, api.BF16)
    assert close_bf16(run(dec, ids, [30] + [1] * 10), want)
    dec.release()


@pytest.mark.parametrize("depth", [1, 2, 3, 4, 5])
def test_layer_by_layer(tmp_path, depth):
    cfg = M.stack()
    cfg["layers"] = cfg["layers"][:depth]
    t = M.tensors(cfg, seed=3)
    ids = tokens(25, cfg["vocab"])
    dec = load(tmp_path, cfg, t)
    assert err(run(dec, ids, []), ref.forward(cfg, t, ids)) <= F32_TOL
    dec.release()


@pytest.mark.parametrize("cuts", [[2] * 60, [3] * 40, [5, 1, 1, 7, 2] * 8, [8] * 15, [64, 2], [119], [1, 119]], ids=str)
@pytest.mark.parametrize("rows", [0, 16])
def test_portions_do_not_change_the_logits(tmp_path, cuts, rows):
    """Also with row blocks of 16, so that a portion is cut again inside and the rings wrap."""
    cfg = M.stack()
    t = M.tensors(cfg, seed=5)
    ids = tokens(120, cfg["vocab"])
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t, block_rows=rows)
    assert err(run(dec, ids, cuts), want) <= F32_TOL
    dec.release()
    dec = load(tmp_path, cfg, t, api.BF16, block_rows=rows)
    assert close_bf16(run(dec, ids, cuts), want)
    dec.release()


def test_portions_on_the_tensor_core_products(tmp_path):
    """bf16: 300 rows take the large-batch products (the experts' too), 5 .. 255 the middle one, 1 .. 4 the row kernel."""
    cfg = M.config([M.layer(heads=4, dim=64, rot_dim=32, vdim=48, kv_rank=96, q_rank=80, window=70, scale=0.1),
                    M.layer(heads=2, dim=128, rot_dim=32, vdim=128, kv_rank=96, q_rank=64, window=150, scale=0.08, kv_from=0, mlp=M.moe(4, 2, 64))], width=128, vocab=200)
    t = M.tensors(cfg, seed=6)
    ids = tokens(310, cfg["vocab"])
    want = ref.forward(cfg, t, ids, np.float32)
    for rows in (0, 130):
        dec = load(tmp_path, cfg, t, api.BF16, max_seq=400, block_rows=rows)
        for cuts in ([300], [128, 64, 100, 5, 4, 2, 1], [290] + [1] * 20):
            assert close_bf16(run(dec, ids, cuts), want, 2e-2)
        dec.release()


def test_first_token_and_the_pair_of_every_portion(tmp_path):
    """The pair table stands out: the row of a sequence's first token, and the previous token over cuts and restarts."""
    cfg = M.config([M.layer(mlp=None)], pairs=(97, 29, 13))
    t = M.tensors(cfg, 4)
    t["bigram"] *= 4.0
    ids = tokens(30, cfg["vocab"], 8)
    want = ref.forward(cfg, t, ids)
    for rows in (0, 4):
        dec = load(tmp_path, cfg, t, block_rows=rows)
        for cuts in ([], [1] * 30, [1, 2, 3, 4, 5, 6], [2] * 15, [29]):
            assert err(run(dec, ids, cuts), want) <= F32_TOL
        assert err(run(dec, ids[5:6], []), ref.forward(cfg, t, ids[5:6])) <= F32_TOL
        dec.release()
    swapped = ref.forward(cfg, t, [ids[1], ids[0]] + ids[2:])
    assert err(swapped[2:3], want[2:3]) > 0.01


def test_a_restart_finds_nothing_of_the_sequence_before(tmp_path):
    cfg = M.stack()
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
    cfg = M.stack()
    t = M.tensors(cfg, seed=8)
    ids = tokens(100, cfg["vocab"])
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t, block_rows=32)
    assert dec.extend(ids[:10], 0).shape == (0, cfg["vocab"])
    pick = [0, 21, 22, 53, 54, 89]
    assert err(dec.extend(ids[10:], 10, pick), want[[10 + p for p in pick]]) <= F32_TOL
    assert err(dec.extend(ids, 0, list(range(100))), want) <= F32_TOL   # more rows than are formed together
    dec.release()


# ---- windows: one key stands out, and the answer depends on whether it is seen ----

SIZES = {"small": {}, "tensor cores": dict(dim=64, vdim=64, rot_dim=32, kv_rank=96)}


@pytest.mark.parametrize("size", sorted(SIZES))
@pytest.mark.parametrize("sources", [0, 1])
@pytest.mark.parametrize("window", [2, 5, 32, 33, 64, 97])
def test_key_just_inside_and_just_outside_the_window(tmp_path, window, sources, size):
    cfg, t = M.needle(window, sources, **SIZES[size])
    rng = np.random.default_rng(window)
    decs = [(load(tmp_path, cfg, t, dt, max_seq=512, block_rows=24), tol) for dt, tol in ((api.F32, F32_TOL), (api.BF16, BF16_TOL))]
    for start in (0, 1, 40):   # where the key lies: the first token, the second, further on
        seen = []
        for distance in (window - 1, window):
            ids = rng.integers(2, 64, start + distance + 4).tolist()
            ids[start] = 1
            ids[start + distance] = 0
            want = ref.forward(cfg, t, ids)
            q = start + distance
            for cuts in ([], [q] + [1] * 4, [max(1, q - 1), 2], [start + 1], [7] * 40):
                for dec, tol in decs:
                    assert err(run(dec, ids, cuts), want) <= tol
            other = list(ids)
            other[start] = 2
            seen.append(err(ref.forward(cfg, t, other)[q:q + 1], want[q:q + 1]))
        assert seen[0] > 0.1 and seen[1] < 1e-9   # inside it decides the answer, outside it is gone
    for dec, _ in decs:
        dec.release()


@pytest.mark.parametrize("sources", [0, 2])
@pytest.mark.parametrize("dtype,tol", [(api.F32, F32_TOL), (api.BF16, BF16_TOL)])
def test_long_decoding_over_rings_that_wrap(tmp_path, dtype, tol, sources):
    """Several hundred decoded tokens; the ring holds window - 1 + 8 positions (its reader's window) and wraps many
    times. The needle is met at the window's edges all along."""
    window = 37
    cfg, t = M.needle(window, sources, heads=3)
    ids = np.random.default_rng(4).integers(2, 64, 420).tolist()
    for p in range(5, 380, 29):
        ids[p] = 1
        ids[p + window - 1 + (p % 2)] = 0
    want = ref.forward(cfg, t, ids)
    dec = load(tmp_path, cfg, t, dtype, max_seq=512, block_rows=8)
    assert err(run(dec, ids, [11] + [1] * 409), want) <= tol
    dec.release()


def test_far_key_over_several_decode_ranges(tmp_path):
    """A window of 300 keys is dealt to several CTAs whose records are merged."""
    cfg, t = M.needle(300, heads=4)
    ids = np.random.default_rng(9).integers(2, 64, 340).tolist()
    ids[3], ids[302], ids[38], ids[337], ids[339] = 1, 0, 1, 0, 0
    want = ref.forward(cfg, t, ids)
    for dtype, tol in ((api.F32, F32_TOL), (api.BF16, BF16_TOL)):
        dec = load(tmp_path, cfg, t, dtype, max_seq=400)
        assert err(run(dec, ids, [295] + [1] * 45), want) <= tol
        assert err(run(dec, ids, []), want) <= tol
        dec.release()


@pytest.mark.parametrize("heads,dim,rot,vdim,kv_rank,window", [(4, 24, 8, 20, 40, 9), (2, 180, 64, 120, 256, 90), (2, 128, 64, 128, 512, 100), (3, 64, 32, 64, 128, 300), (5, 100, 20, 72, 200, 64),
                                                                (8, 64, 64, 128, 64, 1), (2, 32, 128, 96, 96, 2000), (10, 64, 16, 40, 320, 65)])
def test_expanded_and_absorbed_attention_agree(tmp_path, heads, dim, rot, vdim, kv_rank, window):
    """A bf16 decoder's prompt pass (expanded keys and values) against its own decode steps (latents as they are). Queries
    are scaled up so that the softmax is far from uniform."""
    cfg = M.config([M.layer(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=64, window=window, scale=2.0 * (dim + rot) ** -0.5, mlp=None)], width=64, vocab=96)
    t = M.tensors(cfg, seed=heads)
    ids = tokens(330, 96, 2)
    want = ref.forward(cfg, t, ids, np.float32)
    dec = load(tmp_path, cfg, t, api.BF16, max_seq=400, block_rows=150)
    assert err(run(dec, ids, [1] * 330), want) <= 2.5e-2
    for cuts in ([], [40, 111, 33], [200]):
        assert err(run(dec, ids, cuts), want) <= 2.5e-2, cuts
    dec.backend.device_status()
    dec.release()


# ---- generation, sequence keeping, command lines ----

def greedy(cfg, t, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(ref.forward(cfg, t, ids, np.float32)[-1].argmax()))
    return ids[len(prompt):]


def test_greedy_generation(tmp_path):
    cfg = M.stack()
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


def test_replayed_steps_agree_with_the_prompt_pass(tmp_path):
    """bf16: tokens that the captured step generated, fed back as a prompt, give the logits it left behind."""
    cfg = M.stack()
    t = M.tensors(cfg, seed=14)
    prompt = tokens(19, cfg["vocab"])
    dec = load(tmp_path, cfg, t, api.BF16)
    out = dec.complete(prompt, 40)
    left = dec.buffers()[2].cpu().numpy()
    logits = dec.extend(prompt + out[:-1], 0, [len(prompt) + 38])
    assert close_bf16(left[None], logits.astype(np.float64))
    dec.release()


def test_a_sequence_continues_only_where_its_state_is(tmp_path):
    cfg = M.stack()
    dec = load(tmp_path, cfg, M.tensors(cfg, seed=1), max_seq=32)
    dec.extend([1, 2, 3], 0)
    for pos in (1, 2, 4):
        with pytest.raises(api.InvalidArgument):
            dec.extend([4], pos)
    dec.extend([4, 5], 3)
    dec.extend([1] * 27, 5)
    with pytest.raises(api.Unsupported):
        dec.step()
    dec.extend([1], 0)
    dec.release()


def test_configurations_are_checked():
    b = api.gpu_backend()
    good = dict(mixer=MIXER_LATENT, heads=2, dim=8, vdim=8, rot_dims=4, q_rank=8, kv_rank=8, post_norm=True)
    bad = [[dict(good, post_norm=False)], [dict(good, q_rank=0)], [dict(good, kv_rank=0)], [dict(good, rot_dims=3)], [dict(good, vdim=300)], [dict(good, kv_from=0)],
           [dict(good, kv_rank=3000)], [good, dict(good, kv_from=0, kv_rank=16)], [good, dict(good, kv_from=0, rot_base=7.0)], [good, dict(good, kv_from=0), dict(good, kv_from=1)],
           [dict(mixer=MIXER_NONE, post_norm=True)], [dict(mixer=MIXER_NONE, post_norm=True, ffn=8, experts=2)], [dict(mixer=MIXER_NONE, ffn=8)],
           [dict(mixer=9)], [dict(ffn=8, ffn_act=1)]]
    for blocks in bad:
        with pytest.raises(api.TensorError):
            BlockDecoder(b, hidden=64, vocab=10, blocks=[BlockConfig(**x) for x in blocks], max_seq=8)


def test_trace_and_generation_command_lines(tmp_path):
    cfg = M.stack()
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
