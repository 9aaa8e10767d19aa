"""Host-side mirror of the decode loop of the reference's Qwen3 model around the library's
quantized products: Qwen3DecoderLayer / Qwen3Attention / Qwen3MLP forward
(crates/nn-qwen3/src/layers.rs:40-47,94-167,205-226) and the greedy generation loop
(crates/nn-core/src/layers/generation/autoregressive.rs:229-247), for one sequence.

``Decoder`` binds nnq_decoder_* of the C ABI. Weights stay owned by the caller
(``api.DeviceWeight`` / ``api.QuantizedTensor``); token and position live on the device, so
``step`` can be captured in a CUDA graph once and replayed per token (``generate`` does that).

``BlockDecoder`` is the same decoder object made of blocks that each name their own mixer (sliding-window
attention, linear-attention recurrences, attention through a latent, none) and form one residual sum each.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import Callable, List, Optional

import numpy as np

from . import api
from .formats import QuantFormat


class _Config(ctypes.Structure):
    _fields_ = [("hidden", ctypes.c_int32), ("n_heads", ctypes.c_int32), ("n_kv_heads", ctypes.c_int32),
                ("head_dim", ctypes.c_int32), ("ffn", ctypes.c_int32), ("n_layers", ctypes.c_int32),
                ("vocab", ctypes.c_int32), ("max_seq", ctypes.c_int32), ("rms_eps", ctypes.c_float),
                ("rope_theta", ctypes.c_double), ("act_dtype", ctypes.c_int32), ("tp_rank", ctypes.c_int32),
                ("tp_world", ctypes.c_int32)]


@dataclass
class DecoderConfig:
    hidden: int = 4096
    n_heads: int = 32
    n_kv_heads: int = 8
    head_dim: int = 128
    ffn: int = 12288
    n_layers: int = 36
    vocab: int = 151936
    max_seq: int = 2560
    rms_eps: float = 1e-6
    rope_theta: float = 1e6
    act_dtype: int = api.BF16
    tp_rank: int = 0
    tp_world: int = 1


class _DevArray:
    """Device memory of the library seen as an array (torch.as_tensor makes a view of it)."""

    def __init__(self, ptr: int, shape, typestr: str):
        self.__cuda_array_interface__ = {"shape": tuple(shape), "typestr": typestr, "data": (ptr, False), "version": 2}


class Decoder:
    def __init__(self, backend: api.Backend, cfg: DecoderConfig):
        self.backend, self.cfg = backend, cfg
        h = ctypes.c_void_p()
        backend.check(self._create(self._c_config(), ctypes.byref(h)))
        self._handle = h
        self._keep = []   # tensors the library holds pointers to

    def _c_config(self):
        cfg = self.cfg
        return _Config(cfg.hidden, cfg.n_heads, cfg.n_kv_heads, cfg.head_dim, cfg.ffn, cfg.n_layers, cfg.vocab,
                       cfg.max_seq, cfg.rms_eps, cfg.rope_theta, cfg.act_dtype, cfg.tp_rank, cfg.tp_world)

    def _create(self, c_config, out):
        return self.backend._lib.nnq_decoder_create(self.backend._ctx, ctypes.byref(c_config), out)

    def set_layer(self, layer: int, q, k, v, o, gate, up, down, in_norm, post_norm, q_norm, k_norm):
        """Projections: quantized weights; norms: contiguous f32 torch tensors (any device) or numpy arrays."""
        ws = [q, k, v, o, gate, up, down]
        self._keep.extend(ws)
        norms = [self._ptr(t) for t in (in_norm, post_norm, q_norm, k_norm)]
        self.backend.check(self.backend._lib.nnq_decoder_set_layer(self._handle, layer, *[w.handle() for w in ws], *norms))

    def set_head(self, embed_bf16, final_norm, lm_head):
        self._keep.extend([embed_bf16, lm_head])
        self.backend.check(self.backend._lib.nnq_decoder_set_head(self._handle, embed_bf16.data_ptr(), self._ptr(final_norm),
                                                                  lm_head.handle()))

    def set_comm(self, peer):
        """Tensor parallel: the PeerComm whose slots carry the o / down exchanges (max_bytes >= 8 * hidden)."""
        self._keep.append(peer)
        self.backend.check(self.backend._lib.nnq_decoder_set_comm(self._handle, peer._handle))

    @staticmethod
    def _ptr(t):
        if hasattr(t, "data_ptr"):
            return t.data_ptr()
        return t.ctypes.data   # numpy

    def reset(self, token: int, pos: int, stream=None):
        self.backend.check(self.backend._lib.nnq_decoder_reset(self._handle, token, pos, api._stream_ptr(stream)))

    def prefill(self, tokens, start_pos: int = 0, stream=None):
        """Prompt pass over `tokens` (a sequence of ids) at positions start_pos ..: fills the caches,
        leaves the last prompt token's logits and its greedy successor as the next input."""
        arr = np.ascontiguousarray(tokens, dtype=np.int32)
        self.backend.check(self.backend._lib.nnq_decoder_prefill(self._handle, arr.ctypes.data, int(arr.size), int(start_pos),
                                                                 api._stream_ptr(stream)))

    def extend(self, tokens, start_pos: int, want=(), stream=None):
        """Continue the sequence with given tokens at positions start_pos ..; returns the logits (numpy f32
        [len(want), vocab]) after the tokens whose indexes `want` lists in ascending order. One token runs the
        decode step, several run the prompt pass; start_pos 0 starts a new sequence."""
        arr = np.ascontiguousarray(tokens, dtype=np.int32)
        idx = np.ascontiguousarray(want, dtype=np.int32)
        out = np.empty((idx.size, self.cfg.vocab), np.float32)
        self.backend.check(self.backend._lib.nnq_decoder_extend(self._handle, arr.ctypes.data, int(arr.size), int(start_pos),
                                                                idx.ctypes.data, int(idx.size), out.ctypes.data,
                                                                api._stream_ptr(stream)))
        return out

    def step(self, stream=None):
        self.backend.check(self.backend._lib.nnq_decoder_step(self._handle, api._stream_ptr(stream)))

    def step_raw(self, stream_ptr) -> int:
        return self.backend._lib.nnq_decoder_step(self._handle, stream_ptr)

    def state(self, stream=None):
        t, p, n = ctypes.c_int(), ctypes.c_int(), ctypes.c_int()
        self.backend.check(self.backend._lib.nnq_decoder_state(self._handle, ctypes.byref(t), ctypes.byref(p), ctypes.byref(n),
                                                               api._stream_ptr(stream)))
        return t.value, p.value, n.value

    def buffers(self):
        """(key cache, value cache, logits, tokens) as torch views of the library's device memory."""
        import torch
        k, v, lg, tk = ctypes.c_void_p(), ctypes.c_void_p(), ctypes.c_void_p(), ctypes.c_void_p()
        self.backend.check(self.backend._lib.nnq_decoder_buffers(self._handle, ctypes.byref(k), ctypes.byref(v), ctypes.byref(lg),
                                                                 ctypes.byref(tk)))
        c = self.cfg
        dev = torch.device("cuda", self.backend.device)
        shape = (c.n_layers, c.n_kv_heads // c.tp_world, c.max_seq, c.head_dim)
        return (torch.as_tensor(_DevArray(k.value, shape, "<f4"), device=dev),
                torch.as_tensor(_DevArray(v.value, shape, "<f4"), device=dev),
                torch.as_tensor(_DevArray(lg.value, (c.vocab,), "<f4"), device=dev),
                torch.as_tensor(_DevArray(tk.value, (c.max_seq,), "<i4"), device=dev))

    def generate(self, first_token: int, pos: int, n_tokens: int, use_graph: bool = True):
        """Greedy decode of n_tokens starting with `first_token` at position `pos`; returns the
        generated token ids (a list) — one captured graph replayed per token after the first."""
        import torch
        dev = torch.device("cuda", self.backend.device)
        stream = torch.cuda.Stream(device=dev)
        self.reset(first_token, pos, stream)
        with torch.cuda.stream(stream):
            self.step(stream)   # outside a capture: lazy module loading, attribute set-up
            if use_graph and n_tokens > 1:
                stream.synchronize()
                g = torch.cuda.CUDAGraph()
                with torch.cuda.graph(g, stream=stream):
                    self.step(torch.cuda.current_stream())
                for _ in range(n_tokens - 1):
                    g.replay()
            else:
                for _ in range(n_tokens - 1):
                    self.step(stream)
            stream.synchronize()
        self.backend.device_status(stream)
        self.state(stream)   # the library's host side learns the position the replays reached
        toks = self.buffers()[3]
        return toks[pos:pos + n_tokens].cpu().tolist()

    def complete(self, prompt, n_tokens: int, use_graph: bool = True):
        """Greedy continuation of a prompt (token ids) by n_tokens: prompt pass, then the decode loop."""
        prompt = list(prompt)
        self.prefill(prompt, 0)
        first = self.state()[0]
        return [first] + (self.generate(first, len(prompt), n_tokens - 1, use_graph) if n_tokens > 1 else [])

    def release(self):
        if self._handle is not None:
            self.backend._lib.nnq_decoder_destroy(self._handle)
            self._handle = None
            self._keep = []


# --------------------------------------------------------------------------- #
# decoders made of blocks
# --------------------------------------------------------------------------- #

MIXER_ATTENTION, MIXER_RECURRENT, MIXER_LATENT, MIXER_NONE = 0, 1, 2, 3
ACT_SILU, ACT_GELU_TANH = 0, 1


class _BlockConfig(ctypes.Structure):
    _fields_ = [("mixer", ctypes.c_int32), ("heads", ctypes.c_int32), ("kv_heads", ctypes.c_int32), ("dim", ctypes.c_int32),
                ("vdim", ctypes.c_int32), ("ffn", ctypes.c_int32), ("rot_dims", ctypes.c_int32), ("rot_base", ctypes.c_double),
                ("scale", ctypes.c_float), ("window", ctypes.c_int32), ("conv_taps", ctypes.c_int32), ("value_mix", ctypes.c_int32),
                ("out_gate", ctypes.c_int32), ("q_scale", ctypes.c_float), ("k_scale", ctypes.c_float),
                ("decay_rank", ctypes.c_int32), ("decay_tau", ctypes.c_float), ("post_norm", ctypes.c_int32), ("alpha", ctypes.c_float),
                ("ffn_act", ctypes.c_int32), ("experts", ctypes.c_int32), ("q_rank", ctypes.c_int32), ("kv_rank", ctypes.c_int32),
                ("kv_from", ctypes.c_int32)]


class _BlockLayout(ctypes.Structure):
    _fields_ = [(n, ctypes.c_int32) for n in ("in_cols", "in_k", "out_k", "ffn_col", "q", "k", "v", "g", "a1", "gate", "up", "ffn_step",
                                                 "q_ld", "kv_ld", "dim_ld", "vdim_ld")]


class _BlockWeights(ctypes.Structure):
    _fields_ = [("w_in", ctypes.c_void_p), ("w_out", ctypes.c_void_p)] + \
        [(n, ctypes.c_void_p) for n in ("norm", "bias_in", "bias_out", "conv", "head_norm", "decay_w", "decay_b", "decay")] + \
        [("value_lambda", ctypes.c_float)] + \
        [(n, ctypes.c_void_p) for n in ("norm_bias", "uq", "ukv", "q_norm", "kv_norm", "moe")]


class _HeadOptions(ctypes.Structure):
    _fields_ = [("final_norm_bias", ctypes.c_void_p), ("logit_cap", ctypes.c_float), ("pair_table", ctypes.c_void_p),
                ("pair_mul_prev", ctypes.c_int64), ("pair_mul_cur", ctypes.c_int64), ("pair_buckets", ctypes.c_int64)]


@dataclass
class BlockConfig:
    """nnq_block_config of the C ABI; window 0 = every earlier position, decay_rank 0 = a fixed decay per head,
    kv_from < 0 = latents of its own. top and expert_ffn describe a mixture of `experts`."""
    mixer: int = MIXER_ATTENTION
    heads: int = 1
    kv_heads: int = 1
    dim: int = 64
    vdim: int = 64
    ffn: int = 0
    rot_dims: int = 0
    rot_base: float = 1e4
    scale: float = 1.0
    window: int = 0
    conv_taps: int = 0
    value_mix: bool = False
    out_gate: bool = False
    q_scale: float = 1.0
    k_scale: float = 1.0
    decay_rank: int = 0
    decay_tau: float = 1.0
    post_norm: bool = False
    alpha: float = 1.0
    ffn_act: int = ACT_SILU
    experts: int = 0
    q_rank: int = 0
    kv_rank: int = 0
    kv_from: int = -1
    top: int = 0
    expert_ffn: int = 0

    def _c(self) -> _BlockConfig:
        return _BlockConfig(self.mixer, self.heads, self.kv_heads, self.dim, self.vdim, self.ffn, self.rot_dims, self.rot_base,
                            self.scale, self.window, self.conv_taps, int(self.value_mix), int(self.out_gate), self.q_scale,
                            self.k_scale, self.decay_rank, self.decay_tau, int(self.post_norm), self.alpha, self.ffn_act, self.experts,
                            self.q_rank, self.kv_rank, self.kv_from)


@dataclass
class BlockTensors:
    """Tensors of one block: matrices [out, in] as bf16 bit patterns (uint16), everything else f32."""
    norm: np.ndarray
    q: Optional[np.ndarray] = None
    k: Optional[np.ndarray] = None
    v: Optional[np.ndarray] = None
    o: Optional[np.ndarray] = None
    g: Optional[np.ndarray] = None
    q_bias: Optional[np.ndarray] = None
    k_bias: Optional[np.ndarray] = None
    v_bias: Optional[np.ndarray] = None
    o_bias: Optional[np.ndarray] = None
    conv: Optional[np.ndarray] = None        # [channels of q | k | v, taps]
    value_lambda: float = 0.0
    a1: Optional[np.ndarray] = None
    decay_w: Optional[np.ndarray] = None
    decay_b: Optional[np.ndarray] = None
    decay: Optional[np.ndarray] = None       # [heads]
    head_norm: Optional[np.ndarray] = None
    gate: Optional[np.ndarray] = None
    up: Optional[np.ndarray] = None
    down: Optional[np.ndarray] = None
    norm_bias: Optional[np.ndarray] = None
    dq: Optional[np.ndarray] = None          # latent attention: [q_rank, hidden]
    q_norm: Optional[np.ndarray] = None
    uq: Optional[np.ndarray] = None          # [heads * (dim + rot_dims), q_rank]
    dkv: Optional[np.ndarray] = None         # [kv_rank + rot_dims, hidden]
    kv_norm: Optional[np.ndarray] = None
    uk: Optional[np.ndarray] = None          # [heads * dim, kv_rank]
    uv: Optional[np.ndarray] = None          # [heads * vdim, kv_rank]
    router: Optional[np.ndarray] = None      # mixture of experts: f32 [experts, hidden]
    router_bias: Optional[np.ndarray] = None
    expert: Optional[Callable[[int], tuple]] = None   # expert -> (gate, up, down)


class BlockDecoder(Decoder):
    """Decoder whose layers are blocks x <- x + mixer(h) + ff(h), h = RMSNorm(x) * w, or (post_norm) x <- LN(alpha x +
    mixer(x) + ff(x))."""

    def __init__(self, backend: api.Backend, *, hidden: int, vocab: int, blocks: List[BlockConfig], max_seq: int,
                 rms_eps: float = 1e-6, act_dtype: int = api.BF16, block_rows: int = 0):
        self.blocks, self._block_rows = list(blocks), int(block_rows)
        super().__init__(backend, DecoderConfig(hidden=hidden, n_heads=0, n_kv_heads=0, head_dim=0, ffn=0, n_layers=len(blocks),
                                                vocab=vocab, max_seq=max_seq, rms_eps=rms_eps, rope_theta=0.0, act_dtype=act_dtype))

    def _create(self, c_config, out):
        arr = (_BlockConfig * len(self.blocks))(*[b._c() for b in self.blocks])
        return self.backend._lib.nnq_decoder_create_blocks(self.backend._ctx, ctypes.byref(c_config), arr, self._block_rows, out)

    def layout(self, layer: int) -> _BlockLayout:
        y = _BlockLayout()
        self.backend.check(self.backend._lib.nnq_decoder_block_layout(self._handle, layer, ctypes.byref(y)))
        return y

    def _weight(self, rows: int, cols: int, parts) -> api.DeviceWeight:
        """A bf16 weight [rows, cols] of zeros with the given (row, column, matrix) parts, on the device."""
        w = np.zeros((rows, cols), np.uint16)
        for r, c, m in parts:
            if m is not None:
                if r < 0 or r + m.shape[0] > rows or c + m.shape[1] > cols:
                    raise api.ShapeMismatch(f"a matrix of shape {m.shape} does not fit its block")
                w[r:r + m.shape[0], c:c + m.shape[1]] = m
        b, h = self.backend, ctypes.c_void_p()
        b.check(b._lib.nnq_weight_create(b._ctx, int(QuantFormat.BF16_DENSE), w.ctypes.data, w.nbytes, None, 0, rows, cols, ctypes.byref(h)))
        t = api.DeviceWeight(b, h)
        self._keep.append(t)
        return t

    def _heads(self, rows: int, cols: int, parts) -> api.DeviceWeight:
        """A weight made of head-by-head matrices: (first row, rows per head, rows a head is given, matrix) parts."""
        out = []
        for r, per, ld, m in parts:
            out += [(r + h * ld, 0, m[h * per:(h + 1) * per]) for h in range(m.shape[0] // per)]
        return self._weight(rows, cols, out)

    def _experts(self, b: BlockConfig, y: _BlockLayout, t: BlockTensors):
        """The block's experts as a MoeBlock of bf16 weights, widths rounded up to whole k steps with zeros."""
        from .moe import LAYOUT_NK_PAIRS, MoeBlock
        hidden, ld, inter = self.cfg.hidden, y.in_k, -(-b.expert_ffn // 64) * 64
        gu, dn = np.zeros((b.experts, inter, 2, ld), np.uint16), np.zeros((b.experts, ld, inter), np.uint16)
        for e in range(b.experts):
            gate, up, down = t.expert(e)
            if gate.shape != (b.expert_ffn, hidden) or up.shape != gate.shape or down.shape != gate.shape[::-1]:
                raise api.ShapeMismatch(f"expert {e}: matrices of shape {gate.shape}, {up.shape}, {down.shape}")
            gu[e, :b.expert_ffn, 0, :hidden], gu[e, :b.expert_ffn, 1, :hidden], dn[e, :hidden, :b.expert_ffn] = gate, up, down
        router = np.zeros((b.experts, ld), np.float32)
        router[:, :hidden] = t.router
        bias = np.zeros(b.experts, np.float32) if t.router_bias is None else t.router_bias
        m = MoeBlock(b.experts, ld, inter, b.top, float("inf"), router, bias, LAYOUT_NK_PAIRS, QuantFormat.BF16_DENSE,
                     gu.reshape(-1).view(np.uint8), None, None, dn.reshape(-1).view(np.uint8), None, None, self.backend)
        self._keep.append(m)
        return m

    def _set_post(self, layer: int, b: BlockConfig, y: _BlockLayout, t: BlockTensors):
        """Blocks of attention through a latent, of a feed-forward alone or of a mixture of experts."""
        hidden, w = self.cfg.hidden, _BlockWeights()
        want = {"norm": (hidden,), "norm_bias": (hidden,)}
        if b.mixer == MIXER_LATENT:
            want.update(dq=(b.q_rank, hidden), q_norm=(b.q_rank,), uq=(b.heads * (b.dim + b.rot_dims), b.q_rank), uk=(b.heads * b.dim, b.kv_rank),
                        uv=(b.heads * b.vdim, b.kv_rank), o=(hidden, b.heads * b.vdim))
            if b.kv_from < 0:
                want.update(dkv=(b.kv_rank + b.rot_dims, hidden), kv_norm=(b.kv_rank,))
        elif b.experts:
            want.update(router=(b.experts, hidden))
        else:
            want.update(gate=(b.ffn, hidden), up=(b.ffn, hidden), down=(hidden, b.ffn))
        self._check(layer, t, want, {"router_bias": (b.experts,)})
        if b.mixer == MIXER_LATENT:
            w.w_in = self._weight(y.in_cols, y.in_k, [(y.q, 0, t.dq), (y.k, 0, t.dkv if b.kv_from < 0 else None)]).handle()
            w.w_out = self._weight(hidden, y.out_k, [(0, 0, t.o)]).handle()
            w.uq = self._weight(b.heads * (b.dim + b.rot_dims), y.q_ld, [(0, 0, t.uq)]).handle()
            w.ukv = self._heads(b.heads * (y.dim_ld + y.vdim_ld), y.kv_ld,
                                [(0, b.dim, y.dim_ld, t.uk), (b.heads * y.dim_ld, b.vdim, y.vdim_ld, t.uv)]).handle()
        elif b.experts:
            w.moe = self._experts(b, y, t)._handle
        else:
            pairs = np.zeros((y.in_cols, hidden), np.uint16)
            end = y.ffn_step * b.ffn
            pairs[y.gate:end:y.ffn_step], pairs[y.up:end:y.ffn_step] = t.gate, t.up
            w.w_in = self._weight(y.in_cols, y.in_k, [(0, 0, pairs)]).handle()
            w.w_out = self._weight(hidden, y.out_k, [(0, 0, t.down)]).handle()
        f32 = {n: np.ascontiguousarray(getattr(t, n), np.float32) for n in ("norm", "norm_bias", "q_norm", "kv_norm") if getattr(t, n) is not None}
        for n, a in f32.items():
            setattr(w, n, a.ctypes.data)
        self.backend.check(self.backend._lib.nnq_decoder_set_block(self._handle, layer, ctypes.byref(w)))

    @staticmethod
    def _check(layer: int, t: BlockTensors, want: dict, optional: dict):
        for name, shape in list(want.items()) + list(optional.items()):
            a = getattr(t, name)
            if a is None and name in optional:
                continue
            if a is None or tuple(a.shape) != shape:
                raise api.ShapeMismatch(f"block {layer}: {name} must be {shape}, got {None if a is None else tuple(a.shape)}")

    def set_block(self, layer: int, t: BlockTensors):
        y, b, hidden = self.layout(layer), self.blocks[layer], self.cfg.hidden
        if b.mixer in (MIXER_LATENT, MIXER_NONE):
            return self._set_post(layer, b, y, t)
        kvh = b.kv_heads if b.mixer == MIXER_ATTENTION else b.heads
        qn, kn, vn, mix = b.heads * b.dim, kvh * b.dim, kvh * b.vdim, b.heads * b.vdim
        want = {"q": (qn, hidden), "k": (kn, hidden), "v": (vn, hidden), "o": (hidden, mix), "norm": (hidden,)}
        if y.g >= 0:
            want["g"] = (mix, hidden)
        if b.ffn:
            want.update(gate=(b.ffn, hidden), up=(b.ffn, hidden), down=(hidden, b.ffn))
        if b.mixer == MIXER_ATTENTION and b.conv_taps:
            want["conv"] = (qn + kn + vn, b.conv_taps)
        if b.mixer == MIXER_RECURRENT:
            if b.decay_rank:
                want.update(a1=(b.decay_rank, hidden), decay_w=(qn, b.decay_rank), decay_b=(qn,))
            else:
                want["decay"] = (b.heads,)
        optional = {"q_bias": (qn,), "k_bias": (kn,), "v_bias": (vn,), "o_bias": (hidden,), "head_norm": (b.vdim,)}
        if b.post_norm:
            want["norm_bias"] = (hidden,)
        self._check(layer, t, want, optional)
        w_in = self._weight(y.in_cols, y.in_k, [(y.q, 0, t.q), (y.k, 0, t.k), (y.v, 0, t.v), (y.g, 0, t.g), (y.a1, 0, t.a1),
                                                (y.gate, 0, t.gate), (y.up, 0, t.up)])
        w_out = self._weight(hidden, y.out_k, [(0, 0, t.o), (0, y.ffn_col, t.down)])
        bias = None
        if any(x is not None for x in (t.q_bias, t.k_bias, t.v_bias)):
            bias = np.zeros(y.in_cols, np.float32)
            for c, x in ((y.q, t.q_bias), (y.k, t.k_bias), (y.v, t.v_bias)):
                if x is not None:
                    bias[c:c + x.size] = x
        f32 = [None if a is None else np.ascontiguousarray(a, np.float32)
               for a in (t.norm, bias, t.o_bias, t.conv, t.head_norm, t.decay_w, t.decay_b, t.decay)]
        w = _BlockWeights(w_in.handle(), w_out.handle(), *[None if a is None else a.ctypes.data for a in f32], float(t.value_lambda))
        post = np.ascontiguousarray(t.norm_bias, np.float32) if b.post_norm else None
        if b.post_norm:
            w.norm_bias = post.ctypes.data
        self.backend.check(self.backend._lib.nnq_decoder_set_block(self._handle, layer, ctypes.byref(w)))

    def set_head(self, embed, final_norm, lm_head, *, final_norm_bias=None, logit_cap: float = 0.0, pair_table=None, pair_mul=(0, 0)):
        """embed, lm_head: [vocab, hidden] as bf16 bit patterns (uint16); final_norm f32 [hidden], with final_norm_bias a layer
        norm. logit_cap > 0: logits <- cap tanh(logits / cap). pair_table [buckets + 1, hidden] with the factors pair_mul of the
        previous and the current token: the hashed embedding of token pairs."""
        c = self.cfg
        ld = self.layout(0).in_k
        for a in (embed, lm_head):
            if tuple(a.shape) != (c.vocab, c.hidden):
                raise api.ShapeMismatch(f"embedding and vocabulary projection must be {(c.vocab, c.hidden)}, got {tuple(a.shape)}")
        e = self._weight(c.vocab, ld, [(0, 0, embed)])
        h = e if lm_head is embed else self._weight(c.vocab, ld, [(0, 0, lm_head)])
        fn = np.ascontiguousarray(final_norm, np.float32)
        self.backend.check(self.backend._lib.nnq_decoder_set_head_weights(self._handle, e.handle(), fn.ctypes.data, h.handle()))
        o = _HeadOptions(logit_cap=float(logit_cap))
        if final_norm_bias is not None:
            fb = np.ascontiguousarray(final_norm_bias, np.float32)
            o.final_norm_bias = fb.ctypes.data
        if pair_table is not None:
            if pair_table.shape[1] != c.hidden or pair_table.shape[0] < 2:
                raise api.ShapeMismatch(f"pair table of shape {pair_table.shape}")
            o.pair_table = self._weight(pair_table.shape[0], ld, [(0, 0, pair_table)]).handle()
            o.pair_buckets = pair_table.shape[0] - 1
            o.pair_mul_prev, o.pair_mul_cur = (int(m) % o.pair_buckets for m in pair_mul)   # (the row depends on the remainders only)
        self.backend.check(self.backend._lib.nnq_decoder_set_head_options(self._handle, ctypes.byref(o)))

    def set_layer(self, *a, **k):
        raise api.Unsupported("a block decoder takes set_block")

    def buffers(self):
        """(None, None, logits, tokens): the blocks keep their own caches and states."""
        import torch
        lg, tk = ctypes.c_void_p(), ctypes.c_void_p()
        self.backend.check(self.backend._lib.nnq_decoder_buffers(self._handle, None, None, ctypes.byref(lg), ctypes.byref(tk)))
        dev = torch.device("cuda", self.backend.device)
        return (None, None, torch.as_tensor(_DevArray(lg.value, (self.cfg.vocab,), "<f4"), device=dev),
                torch.as_tensor(_DevArray(tk.value, (self.cfg.max_seq,), "<i4"), device=dev))
