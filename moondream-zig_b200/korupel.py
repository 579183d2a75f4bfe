"""The Korupel decoder: reader of its model folder (config.json + model.safetensors) and its description as a layer stack.

config.json
  vocab, width, norm.eps, residual_mult, canon.taps
  layers: a list; each entry has "type" ("attention" or "lightning"), "mixer" and "mlp" (or null)
    attention mixer: heads, kv_heads, dim, vdim (= dim), scale, mask.size, mask.keep_first
    lightning mixer: heads, dim, vdim, decay (one number per head)
    mlp: {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}}
Tensors: embed, head, final.norm, and per layer i "l<i>." + norm1, norm1b, norm2, norm2b, canon1, canon2, mix.*, mlp.*.

A layer's projections that read the same input are one matrix (q | k | g or q | k | v | g), gate and up rows alternate in
blocks of 32, experts are stacked: what the kernels behind md_stack_layer expect.
"""
from __future__ import annotations

import numpy as np

from .models import (ACT_GELU_TANH, ACT_SILU, FF_DENSE, FF_MOE, FF_NONE, MIXER_LIGHTNING, MIXER_WINDOW_ATTENTION,
                     StackModel, down, gate_up, pad_rows as _pad_rows, register_model)

def _per_head(v, heads: int) -> np.ndarray:
    a = np.asarray(v, np.float32).reshape(-1)
    if a.size == 1:
        a = np.repeat(a, heads)
    if a.size != heads:
        raise ValueError(f"{a.size} values for {heads} heads")
    return a


def stack_layers(cfg: dict, t) -> list:
    """One dict per layer for StackModel.  `t(name)` returns a tensor as an array whose bits are kept (matrices) or
    that `StackModel` widens to float32 (vectors)."""
    out = []
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        d = {"norm1": t(p + "norm1"), "norm1b": t(p + "norm1b"), "conv1": t(p + "canon1"),
             "heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"], "w_out": t(p + "mix.o")}
        if layer["type"] == "attention":
            if m["vdim"] != m["dim"]:
                raise ValueError(f"layer {i}: the values are the keys, but vdim {m['vdim']} != dim {m['dim']}")
            mask = m.get("mask") or {}
            q, k, g = t(p + "mix.q"), t(p + "mix.k"), t(p + "mix.g")
            bias = np.concatenate([StackModel.widen(t(p + "mix.q.b")), StackModel.widen(t(p + "mix.k.b")),
                                   np.zeros(g.shape[0], np.float32)])
            d.update(mixer=MIXER_WINDOW_ATTENTION, kv_heads=m["kv_heads"], scale=m["scale"],
                     window=mask.get("size") or 0, keep_first=mask.get("keep_first") or 0, r1=t(p + "mix.r1"),
                     r2=t(p + "mix.r2"), w_in=_pad_rows(np.concatenate([q, k, g]), 8), b_in=_pad_rows(bias, 8))
        elif layer["type"] == "lightning":
            parts = [t(p + "mix." + n) for n in ("q", "k", "v", "g")]
            d.update(mixer=MIXER_LIGHTNING, decay=_per_head(m["decay"], m["heads"]), mix_norm=t(p + "mix.norm"),
                     w_in=_pad_rows(np.concatenate(parts), 8))
        else:
            raise ValueError(f"layer {i}: unknown mixer {layer['type']!r}")
        mlp = layer.get("mlp")
        if mlp is None:
            d["ff"] = FF_NONE
        else:
            d.update(norm2=t(p + "norm2"), norm2b=t(p + "norm2b"), conv2=t(p + "canon2"))
            q = p + "mlp."
            if mlp["kind"] == "dense":
                d.update(ff=FF_DENSE, act=ACT_GELU_TANH, ff_dim=mlp["ff"], w_gate_up=gate_up(t(q + "gate"), t(q + "up")),
                         w_down=down(t(q + "down")))
            elif mlp["kind"] == "moe":
                E = mlp["router"]["experts"]
                d.update(ff=FF_MOE, act=ACT_SILU, ff_dim=mlp["expert"]["ff"], experts=E, top=mlp["router"]["top"],
                         router=t(q + "router"),
                         w_gate_up=np.stack([gate_up(t(f"{q}e{e}.gate"), t(f"{q}e{e}.up")) for e in range(E)]),
                         w_down=np.stack([down(t(f"{q}e{e}.down")) for e in range(E)]))
            else:
                raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
        out.append(d)
    return out


@register_model("Korupel")
def from_tensors(ctx, cfg: dict, tensors, dtype: str = "bfloat16", max_seq: int = 2048) -> StackModel:
    """A model from its configuration and a mapping name -> array (uint16 bfloat16 bits, or floats)."""
    get = tensors.__getitem__
    return StackModel(ctx, stack_layers(cfg, get), embed=get("embed"), head=get("head"), final_norm=get("final.norm"),
                      eps=cfg["norm"]["eps"], residual_mult=cfg["residual_mult"], taps=cfg["canon"]["taps"], dtype=dtype,
                      max_seq=max_seq)
