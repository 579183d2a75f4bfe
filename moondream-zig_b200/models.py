"""ctypes binding of include/moondream_b200_model.h: the device-resident text decoders and
vision encoder built on the hot-path kernels.  Weights are numpy f16 arrays laid out as the
reference holds them (text matrices [out,in], vision matrices [in,out]); they are uploaded
once at construction.

``load_model`` opens a model folder: a config.json names the design in "architecture" and its registered builder reads
model.safetensors; a folder with a moondream.bin gives the Phi-style TextModel.  StackModel is the binding of the
layer-stack decoders (md_stack_weights), which share TextModel's requests, steps and generation."""
from __future__ import annotations

import ctypes as C
import json
import os

import numpy as np

_sz = C.c_size_t

TEXT_PER_LAYER = ("ln_w", "ln_b", "wqkv", "bqkv", "wout", "bout", "wfc1", "bfc1", "wfc2", "bfc2")
TEXT_SINGLE = ("ln_out_w", "ln_out_b", "lm_w", "lm_b", "wte")
VIS_PER_LAYER = ("ln1_w", "ln1_b", "wqkv", "bqkv", "wout", "bout", "ln2_w", "ln2_b", "wfc1", "bfc1", "wfc2", "bfc2")
VIS_SINGLE = ("norm_w", "norm_b", "proj_fc1_w", "proj_fc1_b", "proj_fc2_w", "proj_fc2_b")


class _TextW(C.Structure):
    _fields_ = ([(n, C.c_size_t) for n in ("n_layers", "dim", "hidden", "n_heads", "head_dim", "vocab", "max_seq",
                                           "rot_dim")] +
                [("rope_theta", C.c_float), ("eps_f16", C.c_uint16)] +
                [(n, C.c_void_p) for n in TEXT_PER_LAYER + TEXT_SINGLE])


class _VisW(C.Structure):
    _fields_ = ([(n, C.c_size_t) for n in ("n_layers", "dim", "n_heads", "head_dim", "hidden", "tokens", "patch", "img",
                                           "proj_hidden", "proj_out")] +
                [("eps_f16", C.c_uint16)] +
                [(n, C.c_void_p) for n in ("patch_w", "patch_b", "pos_emb") + VIS_PER_LAYER + VIS_SINGLE])


class _TorchBuf:
    """A CUDA torch tensor used in place of an uploaded weight (kept alive by this wrapper)."""

    def __init__(self, t):
        self.t, self.ptr, self.shape = t, t.data_ptr(), tuple(t.shape)


def _dev(ctx, a):
    """numpy f16 array -> uploaded DevBuf; CUDA torch tensor (f16, contiguous) -> used in place."""
    if hasattr(a, "data_ptr"):
        assert a.is_cuda and a.is_contiguous() and a.element_size() == 2
        return _TorchBuf(a)
    return ctx.upload(np.ascontiguousarray(a, np.float16))


def _f16_bits(v) -> int:
    return int(np.float16(v).view(np.uint16))


class TextRequest:
    """One KVCache (text_model.zig:349) plus the activation buffers of a step."""

    def __init__(self, model: "TextModel"):
        self.model = model
        h = C.c_void_p()
        model.ctx._check(model.lib.md_text_request_create(model.h, C.byref(h)))
        self.h = h

    def reset(self):
        self.model.ctx._check(self.model.lib.md_text_request_reset(self.h))

    def __len__(self):
        n = C.c_size_t()
        self.model.ctx._check(self.model.lib.md_text_request_len(self.h, C.byref(n)))
        return int(n.value)

    def close(self):
        if self.h:
            self.model.lib.md_text_request_destroy(self.h)
            self.h = None


class TextModel:
    logits_dtype = np.float16    # of generate(want_logits=True)

    def __init__(self, ctx, weights: dict, n_heads: int = 32, max_seq: int = 2048, rot_dim: int | None = None,
                 theta: float = 10000.0, eps=np.float16(1e-5)):
        self.ctx, self.lib = ctx, ctx.lib
        self.dev = {}
        s = _TextW()
        L = len(weights["wqkv"])
        dim = weights["wqkv"][0].shape[1]
        s.n_layers, s.dim, s.hidden = L, dim, weights["wfc1"][0].shape[0]
        s.n_heads, s.head_dim = n_heads, dim // n_heads
        s.vocab, s.max_seq = weights["lm_w"].shape[0], max_seq
        s.rot_dim = rot_dim if rot_dim is not None else (dim // n_heads) // 2
        s.rope_theta, s.eps_f16 = theta, _f16_bits(eps)
        self._keep = []
        for name in TEXT_PER_LAYER:
            bufs = [_dev(ctx, a) for a in weights[name]]
            self.dev[name] = bufs
            arr = (C.c_void_p * L)(*[b.ptr for b in bufs])
            self._keep.append(arr)
            setattr(s, name, C.cast(arr, C.c_void_p))
        for name in TEXT_SINGLE:
            b = _dev(ctx, weights[name])
            self.dev[name] = b
            setattr(s, name, b.ptr)
        self._create(s)

    def _create(self, s: _TextW):
        self.s = s
        self.dim, self.vocab, self.n_layers = int(s.dim), int(s.vocab), int(s.n_layers)
        h = C.c_void_p()
        self.ctx._check(self.lib.md_text_model_create(self.ctx.h, C.byref(s), C.byref(h)))
        self.h = h

    @classmethod
    def from_table(cls, ctx, table: _TextW, owner=None) -> "TextModel":
        """A model over weights that are already resident (e.g. a weight file's table); `owner` is kept alive."""
        self = cls.__new__(cls)
        self.ctx, self.lib, self.dev, self._keep = ctx, ctx.lib, {}, [owner]
        self._create(table)
        return self

    def request(self) -> TextRequest:
        return TextRequest(self)

    def text_encoder(self, ids, out_ptr: int | None = None):
        """text_model.zig:106-137.  With out_ptr (a device address) the rows are written there and nothing is returned."""
        ids = np.ascontiguousarray(ids, np.uint32)
        out = np.empty((ids.size, self.dim), np.float16) if out_ptr is None else None
        self.ctx._check(self.lib.md_text_encoder(self.h, C.c_void_p(ids.ctypes.data), _sz(ids.size),
                                                 C.c_void_p(out.ctypes.data if out_ptr is None else out_ptr)))
        return out

    def forward(self, req: TextRequest, embeds, want_hidden=True, want_logits=True, rows: int | None = None):
        """text_decoder + lm_head + argmax over S rows (text_model.zig:139-180,325-345).  embeds: a numpy array
        [S, dim], or a device address together with rows=S."""
        if isinstance(embeds, np.ndarray):
            embeds = np.ascontiguousarray(embeds, np.float16)
            S, src = embeds.shape[0], embeds.ctypes.data
        else:
            S, src = int(rows), int(embeds)
        hidden = np.empty((S, self.dim), np.float16) if want_hidden else None
        logits = np.empty((self.vocab,), np.float16) if want_logits else None
        tok = np.zeros(1, np.uint64)
        self.ctx._check(self.lib.md_text_forward(
            self.h, req.h, C.c_void_p(src), _sz(S),
            C.c_void_p(hidden.ctypes.data if want_hidden else 0), C.c_void_p(logits.ctypes.data if want_logits else 0),
            C.c_void_p(tok.ctypes.data)))
        return hidden, logits, int(tok[0])

    def step(self, req: TextRequest, tokens, want=(), want_token: bool = False):
        """md_text_step: run the next tokens of a request from the state it holds.  Returns (float32 logits
        [len(want), vocab] at the wanted places, argmax of the last row or None)."""
        tokens = np.ascontiguousarray(tokens, np.uint32)
        want = np.ascontiguousarray(want, np.uint32)
        logits = np.empty((want.size, self.vocab), np.float32)
        tok = np.zeros(1, np.uint64)
        self.ctx._check(self.lib.md_text_step(
            self.h, req.h, C.c_void_p(tokens.ctypes.data), _sz(tokens.size), C.c_void_p(want.ctypes.data), _sz(want.size),
            C.c_void_p(logits.ctypes.data if want.size else 0), C.c_void_p(tok.ctypes.data if want_token else 0)))
        return logits, (int(tok[0]) if want_token else None)

    def generate(self, req: TextRequest, first: int, n_steps: int, forced=None, want_logits=False):
        """Greedy decode loop on the device (moondream.zig:323-368)."""
        toks = np.zeros(n_steps, np.uint32)
        f = np.ascontiguousarray(forced, np.uint32) if forced is not None else None
        logits = np.empty((n_steps, self.vocab), self.logits_dtype) if want_logits else None
        self.ctx._check(self.lib.md_text_generate(
            self.h, req.h, C.c_uint32(int(first)), _sz(n_steps), C.c_void_p(toks.ctypes.data),
            C.c_void_p(f.ctypes.data if f is not None else 0), C.c_void_p(logits.ctypes.data if want_logits else 0)))
        return (toks, logits) if want_logits else toks

    def generate_batch(self, reqs, first, n_steps: int, forced=None) -> np.ndarray:
        """Up to 8 requests advanced together; forced [batch, n_steps] = teacher forcing per request."""
        B = len(reqs)
        arr = (C.c_void_p * B)(*[r.h.value for r in reqs])
        f = np.ascontiguousarray(first, np.uint32)
        toks = np.zeros((B, n_steps), np.uint32)
        if forced is None:
            self.ctx._check(self.lib.md_text_generate_batch(self.h, arr, _sz(B), C.c_void_p(f.ctypes.data),
                                                            _sz(n_steps), C.c_void_p(toks.ctypes.data)))
        else:
            fo = np.ascontiguousarray(forced, np.uint32)
            assert fo.shape == (B, n_steps)
            self.ctx._check(self.lib.md_text_generate_batch_forced(self.h, arr, _sz(B), C.c_void_p(f.ctypes.data),
                                                                   _sz(n_steps), C.c_void_p(toks.ctypes.data),
                                                                   C.c_void_p(fo.ctypes.data)))
        return toks

    def close(self):
        if getattr(self, "h", None):
            self.lib.md_text_model_destroy(self.h)
            self.h = None


# ---------------------------------------------------------------- layer-stack decoders

DTYPES = {"bfloat16": 1, "float32": 2}
MIXER_WINDOW_ATTENTION, MIXER_LIGHTNING, MIXER_LATENT_ATTENTION = 1, 2, 3
FF_NONE, FF_DENSE, FF_MOE = 0, 1, 2
ACT_GELU_TANH, ACT_SILU, ACT_CLAMPED = 1, 2, 3
LAYER_SANDWICH, LAYER_PARALLEL = 0, 1
ROUTER_LOGISTIC, ROUTER_SOFTMAX = 0, 1


GLU_BLOCK = 32


def pad_rows(a: np.ndarray, multiple: int) -> np.ndarray:
    short = -a.shape[0] % multiple
    return np.concatenate([a, np.zeros((short,) + a.shape[1:], a.dtype)]) if short else a


def gate_up(gate: np.ndarray, up: np.ndarray) -> np.ndarray:
    """[ff, K] x 2 -> [2 * ff_pad, K]: blocks of 32 gate rows and the 32 up rows beside them."""
    gate, up = pad_rows(gate, GLU_BLOCK), pad_rows(up, GLU_BLOCK)
    k = gate.shape[1]
    return np.stack([gate.reshape(-1, GLU_BLOCK, k), up.reshape(-1, GLU_BLOCK, k)], 1).reshape(-1, k)


def down(w: np.ndarray) -> np.ndarray:
    """[width, ff] -> [width, ff_pad]."""
    return np.ascontiguousarray(pad_rows(w.T, GLU_BLOCK).T)


class _StackLayer(C.Structure):
    _fields_ = ([(n, C.c_int) for n in ("mixer", "ff")] +
                [(n, C.c_size_t) for n in ("heads", "kv_heads", "dim", "vdim", "window", "keep_first")] +
                [("scale", C.c_float)] + [(n, C.c_void_p) for n in ("r1", "r2", "decay", "mix_norm", "w_in", "b_in")] +
                [("in_rows", C.c_size_t)] +
                [(n, C.c_void_p) for n in ("w_out", "norm1", "norm1b", "norm2", "norm2b", "conv1", "conv2")] +
                [("act", C.c_int), ("ff_dim", C.c_size_t), ("ff_pad", C.c_size_t)] +
                [(n, C.c_void_p) for n in ("w_gate_up", "w_down", "router")] +
                [("experts", C.c_size_t), ("top", C.c_size_t), ("form", C.c_int), ("router_kind", C.c_int), ("ls1", C.c_void_p),
                 ("ls2", C.c_void_p), ("act_limit", C.c_float), ("act_alpha", C.c_float), ("shared_ff", C.c_size_t),
                 ("shared_pad", C.c_size_t), ("shared_limit", C.c_float), ("shared_gate_up", C.c_void_p),
                 ("shared_down", C.c_void_p), ("q_rank", C.c_size_t), ("kv_rank", C.c_size_t), ("rot_dim", C.c_size_t),
                 ("rope_base", C.c_float)] +
                [(n, C.c_void_p) for n in ("q_norm", "kv_norm", "sink", "w_uq", "w_ukv", "w_ukt")])


class _StackW(C.Structure):
    _fields_ = ([("dtype", C.c_int)] + [(n, C.c_size_t) for n in ("n_layers", "width", "vocab", "max_seq", "taps")] +
                [("eps", C.c_float), ("residual_mult", C.c_float)] +
                [(n, C.c_void_p) for n in ("layers", "embed", "head", "final_norm")])


class StackModel(TextModel):
    """A text model described layer by layer (md_stack_model_create).  `layers`: one dict per layer with the fields of
    md_stack_layer; arrays may be numpy (uint16 = bfloat16 bits, or floats) or CUDA torch tensors already of the model's
    type, which are used in place.  An array that several layers name is uploaded once.  head None: the embedding table."""
    logits_dtype = np.float32
    VECTORS = ("r1", "r2", "decay", "mix_norm", "b_in", "norm1", "norm1b", "norm2", "norm2b", "conv1", "conv2", "ls1", "ls2",
               "q_norm", "kv_norm", "sink")
    MATRICES = ("w_in", "w_out", "w_gate_up", "w_down", "router", "shared_gate_up", "shared_down", "w_uq", "w_ukv", "w_ukt")
    SIZES = ("kv_heads", "window", "keep_first", "act", "ff_dim", "experts", "top", "form", "router_kind", "shared_ff", "q_rank",
             "kv_rank", "rot_dim")
    FLOATS = ("scale", "act_limit", "act_alpha", "shared_limit", "rope_base")

    def __init__(self, ctx, layers: list, embed, head, final_norm, eps: float, residual_mult: float = 1.0, taps: int = 1,
                 dtype: str = "bfloat16", max_seq: int = 2048):
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r}: expected one of {sorted(DTYPES)}")
        self.ctx, self.lib, self.dtype = ctx, ctx.lib, dtype
        self.dev, self._keep, self._bufs, self._uploaded = {}, [], [], {}
        table = (_StackLayer * len(layers))()
        for s, d in zip(table, layers):
            for n in ("mixer", "ff", "heads", "dim", "vdim"):
                setattr(s, n, int(d[n]))
            for n in self.SIZES:
                setattr(s, n, int(d.get(n) or 0))
            for n in self.FLOATS:
                setattr(s, n, float(d.get(n) or 0.0))
            s.in_rows = d["w_in"].shape[0]
            if d["ff"] != FF_NONE:
                s.ff_pad = d["w_down"].shape[-1]
            if d.get("shared_ff"):
                s.shared_pad = d["shared_down"].shape[-1]
            for n in self.VECTORS:
                if d.get(n) is not None:
                    setattr(s, n, self._once(self._vector, d[n], n.startswith("conv")))
            for n in self.MATRICES:
                if d.get(n) is not None:
                    setattr(s, n, self._once(self._matrix, d[n]))
        w = _StackW()
        w.dtype, w.n_layers, w.width, w.vocab, w.max_seq, w.taps = (DTYPES[dtype], len(layers), embed.shape[1],
                                                                    embed.shape[0], max_seq, taps)
        w.eps, w.residual_mult = eps, residual_mult
        w.layers = C.cast(table, C.c_void_p)
        w.embed = self._matrix(embed)
        w.head, w.final_norm = w.embed if head is None else self._matrix(head), self._vector(final_norm)
        self.s = w
        self.dim, self.vocab, self.n_layers = int(w.width), int(w.vocab), int(w.n_layers)
        h = C.c_void_p()
        ctx._check(self.lib.md_stack_model_create(ctx.h, C.byref(w), C.byref(h)))
        self.h = h
        self._uploaded = {}

    def _once(self, upload, a, transposed: bool = False):
        """Device address of an array that several layers may share."""
        key = (id(a), upload.__name__, transposed)
        if key not in self._uploaded:
            self._uploaded[key] = (upload(a.T if transposed else a), a)   # the reference keeps the id in use
        return self._uploaded[key][0]

    @staticmethod
    def widen(a: np.ndarray) -> np.ndarray:
        """bfloat16 bits (uint16) or floats -> float32."""
        a = np.ascontiguousarray(a)
        if a.dtype == np.uint16:
            return (a.astype(np.uint32) << 16).view(np.float32)
        return a.astype(np.float32)

    @staticmethod
    def narrow(a: np.ndarray) -> np.ndarray:
        """bfloat16 bits as they are, floats rounded to nearest even."""
        a = np.ascontiguousarray(a)
        if a.dtype == np.uint16:
            return a
        u = a.astype(np.float32).view(np.uint32)
        return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)

    def _upload(self, a):
        if hasattr(a, "data_ptr"):
            assert a.is_cuda and a.is_contiguous()
            b = _TorchBuf(a)
        else:
            b = self.ctx.upload(a)
        self._bufs.append(b)
        return b.ptr

    def _matrix(self, a):
        if hasattr(a, "data_ptr"):
            assert a.element_size() == (4 if self.dtype == "float32" else 2)
            return self._upload(a)
        return self._upload(self.widen(a) if self.dtype == "float32" else self.narrow(a))

    def _vector(self, a):
        if hasattr(a, "data_ptr"):
            return self._upload(a.float().contiguous())
        return self._upload(self.widen(a))

    def layer_stream(self, req: TextRequest, layer: int, rows: int) -> np.ndarray:
        """Residual stream after `layer` of the last step (set the option "stack_trace" before it)."""
        out = np.empty((rows, self.dim), np.float32)
        self.ctx._check(self.lib.md_text_layer_stream(req.h, _sz(layer), C.c_void_p(out.ctypes.data), _sz(rows)))
        return out

    def close(self):
        super().close()
        for b in self._bufs:
            if not isinstance(b, _TorchBuf):
                self.ctx.release(b)
        self._bufs = []


# architecture name of a config.json -> builder(ctx, config, tensors, dtype=, max_seq=)
MODELS: dict = {}


def register_model(name: str):
    def add(fn):
        MODELS[name] = fn
        return fn
    return add


def load_model(ctx, folder: str, dtype: str = "bfloat16", max_seq: int = 2048):
    """The text model of a folder: config.json + model.safetensors of a registered architecture, or moondream.bin."""
    from . import korupel, nuvezen, weights  # noqa: F401  (each design registers its architecture)
    path = os.path.join(folder, "config.json")
    if not os.path.exists(path) and os.path.exists(os.path.join(folder, "moondream.bin")):
        return weights.WeightFile(os.path.join(folder, "moondream.bin")).upload(ctx).text_model()
    with open(path) as f:
        cfg = json.load(f)
    name = cfg.get("architecture")
    if name not in MODELS:
        raise ValueError(f"architecture {name!r} is not one of {sorted(MODELS)}")
    with weights.SafetensorsFile(os.path.join(folder, "model.safetensors")) as tensors:
        return MODELS[name](ctx, cfg, tensors, dtype=dtype, max_seq=max_seq)


class RequestPool:
    """Requests of one model that are reused: a finished request's caches and states serve the next one."""

    def __init__(self, model: TextModel):
        self.model, self.free, self.live = model, [], {}

    def get(self, key) -> TextRequest:
        if key not in self.live:
            if self.free:
                r = self.free.pop()
                r.reset()
            else:
                r = self.model.request()
            self.live[key] = r
        return self.live[key]

    def end(self, key):
        self.free.append(self.live.pop(key))

    def close(self):
        for r in self.free + list(self.live.values()):
            r.close()
        self.free, self.live = [], {}


class VisionModel:
    def __init__(self, ctx, weights: dict, n_heads: int = 16, img: int = 378, patch: int = 14, max_crops: int = 2,
                 eps=np.float16(1e-5)):
        self.ctx, self.lib = ctx, ctx.lib
        self.dev = {}
        s = _VisW()
        L = len(weights["wqkv"])
        s.n_layers, s.dim = L, weights["wqkv"][0].shape[0]
        s.n_heads, s.head_dim = n_heads, s.dim // n_heads
        s.hidden = weights["wfc1"][0].shape[1]
        s.tokens, s.patch, s.img = weights["pos_emb"].shape[0], patch, img
        s.proj_hidden, s.proj_out = weights["proj_fc1_w"].shape[1], weights["proj_fc2_w"].shape[1]
        s.eps_f16 = _f16_bits(eps)
        self._keep = []
        for name in VIS_PER_LAYER:
            bufs = [_dev(ctx, a) for a in weights[name]]
            self.dev[name] = bufs
            arr = (C.c_void_p * L)(*[b.ptr for b in bufs])
            self._keep.append(arr)
            setattr(s, name, C.cast(arr, C.c_void_p))
        for name in ("patch_w", "patch_b", "pos_emb") + VIS_SINGLE:
            b = _dev(ctx, weights[name])
            self.dev[name] = b
            setattr(s, name, b.ptr)
        self._create(s, max_crops)

    def _create(self, s: _VisW, max_crops: int):
        self.s = s
        self.tokens, self.dim, self.proj_out, self.img = int(s.tokens), int(s.dim), int(s.proj_out), int(s.img)
        self.max_crops = int(max_crops)
        h = C.c_void_p()
        self.ctx._check(self.lib.md_vision_model_create(self.ctx.h, C.byref(s), _sz(max_crops), C.byref(h)))
        self.h = h

    @classmethod
    def from_table(cls, ctx, table: _VisW, max_crops: int = 2, owner=None) -> "VisionModel":
        self = cls.__new__(cls)
        self.ctx, self.lib, self.dev, self._keep = ctx, ctx.lib, {}, [owner]
        self._create(table, max_crops)
        return self

    def encode(self, crops_u8: np.ndarray, crop_a: int = 0, crop_b: int | None = None, want_features: bool = False,
               out_ptr: int | None = None):
        """vision_model.zig:160-202 without the file decode. crops uint8 [c, img, img, 3].  With out_ptr (a device
        address) the [tokens, proj_out] result stays on the device and nothing is returned."""
        crops_u8 = np.ascontiguousarray(crops_u8, np.uint8)
        c = crops_u8.shape[0]
        crop_b = min(1, c - 1) if crop_b is None else crop_b
        feats = np.empty((c * self.tokens, self.dim), np.float16) if want_features else None
        out = np.empty((self.tokens, self.proj_out), np.float16) if out_ptr is None else None
        self.ctx._check(self.lib.md_vision_encode(self.h, C.c_void_p(crops_u8.ctypes.data), _sz(c), _sz(crop_a),
                                                  _sz(crop_b), C.c_void_p(feats.ctypes.data if want_features else 0),
                                                  C.c_void_p(out.ctypes.data if out_ptr is None else out_ptr)))
        return (out, feats) if want_features else out

    def encode_images(self, images_u8: np.ndarray, out_ptrs=None):
        """n independent one-crop images in one pass (md_vision_encode_images).  images uint8 [n, img, img, 3].
        out_ptrs: n device addresses of [tokens, proj_out] buffers; without them a numpy array [n, tokens, proj_out]
        is returned."""
        images_u8 = np.ascontiguousarray(images_u8, np.uint8)
        n = images_u8.shape[0]
        out = None
        if out_ptrs is None:
            out = np.empty((n, self.tokens, self.proj_out), np.float16)
            out_ptrs = [out[i].ctypes.data for i in range(n)]
        arr = (C.c_void_p * n)(*[int(p) for p in out_ptrs])
        self.ctx._check(self.lib.md_vision_encode_images(self.h, C.c_void_p(images_u8.ctypes.data), _sz(n), arr))
        return out

    def close(self):
        if getattr(self, "h", None):
            self.lib.md_vision_model_destroy(self.h)
            self.h = None
