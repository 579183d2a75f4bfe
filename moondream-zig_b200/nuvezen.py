"""The Nuvezen decoder: reader of its model folder (config.json + model.safetensors) and its description as a layer stack.

config.json
  vocab, width, norm.eps
  layers: a list; each entry has "type" ("latent_attention"), "mixer", "mlp" (or null) and, for a layer that runs another
  layer's weights with a cache of its own, "weights_of"
    mixer: heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, mask.size, rot.base, rot.dims (= rot_dim)
    mlp: {"kind": "dense", "ff"} or {"kind": "moe", "expert": {"ff", "limit"}, "router": {"experts", "top"},
         "shared": {"ff", "limit"}}
Tensors: embed (also the head), final.norm, and per layer i that owns its weights "l<i>." + norm1, norm2, ls1, ls2, mix.*, mlp.*.

A layer is parallel: x += ls1 * mixer(norm1(x)) + ls2 * ff(norm2(x)).  The layers' norm weights are stored around zero, the
latents' are plain.  The query's and the keys' projections into their latents are one matrix, a router carries the shared
expert's gate as its last row, gate and up rows alternate in blocks of 32, experts are stacked: what the kernels behind
md_stack_layer expect.
"""
from __future__ import annotations

import numpy as np

from .models import (ACT_CLAMPED, ACT_SILU, FF_DENSE, FF_MOE, FF_NONE, LAYER_PARALLEL, MIXER_LATENT_ATTENTION, ROUTER_SOFTMAX,
                     StackModel, down, gate_up, pad_rows, register_model)

GATE_SLOPE = 1.702      # of the experts' clamped gate


def owner(layers: list, i: int) -> int:
    """The layer whose tensors layer i uses."""
    seen = set()
    while layers[i].get("weights_of") is not None:
        if i in seen:
            raise ValueError(f"layer {i}: weights_of runs in a circle")
        seen.add(i)
        i = layers[i]["weights_of"]
    return i


def norm_weight(w) -> np.ndarray:
    """A weight stored around zero, as the factor it stands for."""
    return np.float32(1.0) + StackModel.widen(w)


def _mixer(i: int, m: dict, t, p: str) -> dict:
    H, d, rot, e, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    rotation = m["rot"]
    if rotation["dims"] != rot:
        raise ValueError(f"layer {i}: rot.dims {rotation['dims']} != rot_dim {rot}")
    uk, uv = t(p + "uk"), t(p + "uv")
    for name, a, shape in (("uq", t(p + "uq"), (H * (d + rot), m["q_rank"])), ("uk", uk, (H * d, R)), ("uv", uv, (H * e, R))):
        if a.shape != shape:
            raise ValueError(f"layer {i}: {name} is {a.shape}, expected {shape}")
    return {"mixer": MIXER_LATENT_ATTENTION, "heads": H, "dim": d, "vdim": e, "rot_dim": rot, "q_rank": m["q_rank"], "kv_rank": R,
            "scale": m["scale"], "window": (m.get("mask") or {}).get("size") or 0, "rope_base": rotation["base"],
            "w_in": pad_rows(np.concatenate([t(p + "dq"), t(p + "dkv")]), 8), "w_out": t(p + "o"), "w_uq": t(p + "uq"),
            "w_ukv": np.concatenate([uk, uv]), "w_ukt": np.ascontiguousarray(uk.reshape(H, d, R).transpose(0, 2, 1)),
            "q_norm": t(p + "dq.norm"), "kv_norm": t(p + "dkv.norm"), "sink": t(p + "sink")}


def _feed_forward(i: int, mlp: dict | None, t, p: str) -> dict:
    if mlp is None:
        return {"ff": FF_NONE}
    if mlp["kind"] == "dense":
        return {"ff": FF_DENSE, "act": ACT_SILU, "ff_dim": mlp["ff"], "w_gate_up": gate_up(t(p + "gate"), t(p + "up")),
                "w_down": down(t(p + "down"))}
    if mlp["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {mlp['kind']!r}")
    E, shared = mlp["router"]["experts"], mlp.get("shared")
    router = t(p + "router")
    d = {"ff": FF_MOE, "act": ACT_CLAMPED, "act_limit": mlp["expert"]["limit"], "act_alpha": GATE_SLOPE, "ff_dim": mlp["expert"]["ff"],
         "experts": E, "top": mlp["router"]["top"], "router_kind": ROUTER_SOFTMAX,
         "w_gate_up": np.stack([gate_up(t(f"{p}e{e}.gate"), t(f"{p}e{e}.up")) for e in range(E)]),
         "w_down": np.stack([down(t(f"{p}e{e}.down")) for e in range(E)])}
    if shared:
        router = np.concatenate([router, t(p + "shared.sg").reshape(1, -1)])
        d.update(shared_ff=shared["ff"], shared_limit=shared["limit"], shared_gate_up=gate_up(t(p + "shared.gate"), t(p + "shared.up")),
                 shared_down=down(t(p + "shared.down")))
    d["router"] = router
    return d


def stack_layers(cfg: dict, t) -> list:
    """One dict per layer for StackModel.  `t(name)` returns a tensor as an array whose bits are kept (matrices) or that
    `StackModel` widens to float32 (vectors).  Layers that share weights hold the same arrays."""
    layers, out, own = cfg["layers"], [], {}
    for i, layer in enumerate(layers):
        j = owner(layers, i)
        if j not in own:
            if layers[j]["type"] != "latent_attention":
                raise ValueError(f"layer {j}: unknown mixer {layers[j]['type']!r}")
            p = f"l{j}."
            d = {"form": LAYER_PARALLEL, "norm1": norm_weight(t(p + "norm1")), "ls1": t(p + "ls1")}
            d.update(_mixer(j, layers[j]["mixer"], t, p + "mix."))
            d.update(_feed_forward(j, layers[j].get("mlp"), t, p + "mlp."))
            if d["ff"] != FF_NONE:
                d.update(norm2=norm_weight(t(p + "norm2")), ls2=t(p + "ls2"))
            own[j] = d
        out.append(own[j])
    return out


@register_model("Nuvezen")
def from_tensors(ctx, cfg: dict, tensors, dtype: str = "bfloat16", max_seq: int = 2048) -> StackModel:
    """A model from its configuration and a mapping name -> array (uint16 bfloat16 bits, or floats)."""
    get = tensors.__getitem__
    return StackModel(ctx, stack_layers(cfg, get), embed=get("embed"), head=None, final_norm=norm_weight(get("final.norm")),
                      eps=cfg["norm"]["eps"], dtype=dtype, max_seq=max_seq)
