"""Small synthetic Korupel models for the tests: configurations of deliberately odd and of kernel-friendly sizes."""
import json
import struct

import numpy as np

import korupel_reference as ref


def attention(heads, kv_heads, dim, size, keep_first, mlp, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5,
                      "mask": {"size": size, "keep_first": keep_first}}}


def lightning(heads, dim, vdim, mlp, decay=None):
    decay = list(decay if decay is not None else np.linspace(0.55, 0.995, heads))
    return {"type": "lightning", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, taps, layers, eps=1e-5, mult=0.7):
    return {"architecture": "Korupel", "width": width, "vocab": vocab, "canon": {"taps": taps}, "norm": {"eps": eps},
            "residual_mult": mult, "layers": layers}


CONFIGS = {
    # every branch, sizes that no fast path can take whole
    "odd": config(90, 61, 4, [attention(6, 2, 14, 7, 2, dense(40)), lightning(3, 10, 22, moe(5, 2, 24)),
                              attention(3, 3, 30, 16, 0, None), lightning(2, 33, 7, dense(50)),
                              attention(4, 1, 18, 5, 9, moe(4, 4, 11))], eps=3e-4, mult=1.3),
    # values that are 1 or equal: one tap, one expert per token, a window of one key, one head, width = head size
    "ones": config(32, 40, 1, [attention(1, 1, 32, 1, 1, moe(3, 1, 32)), lightning(1, 32, 32, dense(32), decay=[1.0]),
                               attention(2, 2, 16, 3, 0, dense(64)), lightning(2, 1, 1, None, decay=[0.0, 0.5])], eps=0.05, mult=1.0),
    # multiples of 8 and 16: the tensor-core and vector paths
    "even": config(192, 136, 3, [lightning(3, 64, 48, dense(320)), attention(8, 2, 64, 100, 5, moe(16, 3, 64)),
                                 lightning(4, 32, 64, moe(9, 4, 96)), attention(6, 1, 80, 33, 1, dense(128))]),
    # larger heads and groups, long recurrences
    "wide": config(512, 264, 2, [attention(16, 1, 128, 70, 3, moe(24, 6, 128)), lightning(4, 128, 128, moe(12, 2, 160)),
                                 attention(4, 4, 112, 200, 0, dense(512)), lightning(2, 96, 160, dense(256))]),
}


def make(name, seed=1):
    cfg = CONFIGS[name]
    return cfg, ref.random_weights(cfg, seed)


def tokens(cfg, n, seed=0):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n)


def rel_err(got, want):
    """Per row: rms of the difference (mean over the vocabulary taken off) over the rms spread of the expected rows."""
    d = np.asarray(got, np.float64) - want
    d = d - d.mean(-1, keepdims=True)
    w = want - want.mean(-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())


LIMITS = {"float32": 5e-5, "bfloat16": 0.1}


def assert_logits(got, want, dtype, what=""):
    e = rel_err(got, want)
    assert np.isfinite(np.asarray(got)).all(), what
    over = int((e > LIMITS[dtype]).sum())
    assert over == 0, f"{what}: {over} of {e.size} rows over {LIMITS[dtype]}, worst {e.max():.3e}, first {np.nonzero(e > LIMITS[dtype])[0][:8]}"


def bits(a):
    return (np.ascontiguousarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)


def write_folder(path, cfg, w):
    """config.json + model.safetensors (bfloat16) as a user's model folder holds them."""
    header, blobs, at = {}, [], 0
    for name, a in w.items():
        b = bits(a).tobytes()
        header[name] = {"dtype": "BF16", "shape": list(a.shape), "data_offsets": [at, at + len(b)]}
        at += len(b)
        blobs.append(b)
    h = json.dumps(header).encode()
    with open(path / "model.safetensors", "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    (path / "config.json").write_text(json.dumps(cfg))
