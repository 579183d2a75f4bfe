"""Plain, slow restatement of the Nuvezen decoder in numpy float64: one function per mechanism, whole sequences, no cache.
Test infrastructure; it shares no code with the library.

Weights are a dict name -> array; names and the meaning of the configuration are those of the model folder a user loads
(config.json + model.safetensors).
"""
import numpy as np


def f64(a):
    return np.asarray(a, np.float64)


def unit_rms(x, eps):
    x = f64(x)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    """RMS norm with a plain weight (the latents)."""
    return unit_rms(x, eps) * f64(w)


def rms_norm_zero(x, w, eps):
    """RMS norm whose weight is stored around zero (the layers and the end of the stack)."""
    return unit_rms(x, eps) * (1.0 + f64(w))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-f64(z)))


def silu(z):
    return f64(z) * sigmoid(z)


def rotate(x, pos, base):
    """x [T, ..., R]: pair (2 i, 2 i + 1) of the last axis turned by pos * base^(-2 i / R)."""
    x = f64(x)
    R = x.shape[-1]
    f = float(base) ** (-np.arange(0, R, 2, dtype=np.float64) / R)
    a = f64(pos)[:, None] * f
    a = a.reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (R // 2,))
    u, v = x[..., 0::2], x[..., 1::2]
    y = np.empty_like(x)
    y[..., 0::2] = u * np.cos(a) - v * np.sin(a)
    y[..., 1::2] = v * np.cos(a) + u * np.sin(a)
    return y


def visible(i, j, size):
    """size 0: every earlier token."""
    return 0 <= i - j and (not size or i - j < size)


def sink_softmax(s, sink):
    """Weights over the last axis; exp(sink) joins the denominator.  Masked scores are -inf."""
    s = f64(s)
    m = np.maximum(s.max(-1), sink)[..., None]
    e = np.exp(s - m)
    return e / (e.sum(-1, keepdims=True) + np.exp(sink - m))


def latents(h, w, pre, kv_rank, eps):
    """Query latent, key/value latent (both normed) and the shared rotated key part before its rotation."""
    cq = rms_norm(h @ f64(w[pre + "dq"]).T, w[pre + "dq.norm"], eps)
    kv = h @ f64(w[pre + "dkv"]).T
    return cq, rms_norm(kv[:, :kv_rank], w[pre + "dkv.norm"], eps), kv[:, kv_rank:]


def latent_attention(cq, c, kr, w, pre, m):
    """Heads' outputs [T, H * vdim] from the latents of a whole sequence."""
    T, H, d, r, e = cq.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = np.arange(T)
    q = (cq @ f64(w[pre + "uq"]).T).reshape(T, H, d + r)
    qr = rotate(q[..., d:], pos, m["rot"]["base"])
    kr = rotate(kr, pos, m["rot"]["base"])
    k = (c @ f64(w[pre + "uk"]).T).reshape(T, H, d)
    v = (c @ f64(w[pre + "uv"]).T).reshape(T, H, e)
    size = (m.get("mask") or {}).get("size") or 0
    dist = pos[:, None] - pos[None, :]
    mask = (dist >= 0) & ((dist < size) if size else True)
    out = np.zeros((T, H, e))
    for h in range(H):
        s = (q[:, h, :d] @ k[:, h].T + qr[:, h] @ kr.T) * m["scale"]
        out[:, h] = sink_softmax(np.where(mask, s, -np.inf), float(f64(w[pre + "sink"])[h])) @ v[:, h]
    return out.reshape(T, H * e)


def mixer(h, m, w, pre, eps):
    cq, c, kr = latents(h, w, pre, m["kv_rank"], eps)
    return latent_attention(cq, c, kr, w, pre, m) @ f64(w[pre + "o"]).T


def silu_ff(h, gate, up, down):
    return (silu(h @ f64(gate).T) * (h @ f64(up).T)) @ f64(down).T


def clamped_ff(h, gate, up, down, limit):
    g = np.minimum(h @ f64(gate).T, limit)
    u = np.clip(h @ f64(up).T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ f64(down).T


def route(h, router, top):
    """Indices of the `top` largest logits per token and the softmax over those alone."""
    z = h @ f64(router).T
    sel = np.argsort(-z, axis=-1, kind="stable")[:, :top]
    zc = np.take_along_axis(z, sel, -1)
    p = np.exp(zc - zc.max(-1, keepdims=True))
    return sel, p / p.sum(-1, keepdims=True)


def moe_ff(h, mlp, w, pre):
    r, ex = mlp["router"], mlp["expert"]
    sel, p = route(h, w[pre + "router"], r["top"])
    y = np.zeros_like(f64(h))
    for e in range(r["experts"]):
        rows, slot = np.nonzero(sel == e)
        if rows.size:
            y[rows] += p[rows, slot][:, None] * clamped_ff(h[rows], w[f"{pre}e{e}.gate"], w[f"{pre}e{e}.up"],
                                                           w[f"{pre}e{e}.down"], ex["limit"])
    if mlp.get("shared"):
        y += shared_ff(h, mlp["shared"], w, pre + "shared.")
    return y


def shared_ff(h, shared, w, pre):
    y = clamped_ff(h, w[pre + "gate"], w[pre + "up"], w[pre + "down"], shared["limit"])
    return y * sigmoid(h @ f64(w[pre + "sg"]).T)


def feed_forward(h, mlp, w, pre):
    if mlp["kind"] == "dense":
        return silu_ff(h, w[pre + "gate"], w[pre + "up"], w[pre + "down"])
    return moe_ff(h, mlp, w, pre)


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def layer_step(x, layer, w, p, eps):
    """Both sublayers read the same x."""
    y = f64(w[p + "ls1"]) * mixer(rms_norm_zero(x, w[p + "norm1"], eps), layer["mixer"], w, p + "mix.", eps)
    if layer["mlp"] is not None:
        y = y + f64(w[p + "ls2"]) * feed_forward(rms_norm_zero(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.")
    return x + y


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    embed = f64(w["embed"])
    x = embed[np.asarray(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        x = layer_step(x, layer, w, f"l{owner(cfg, i)}.", eps)
        streams.append(x)
    logits = rms_norm_zero(x, w["final.norm"], eps) @ embed.T
    return (logits, np.stack(streams)) if want_layers else logits


# ---------------------------------------------------------------- synthetic models for the tests

def to_bf16(a):
    """Round to bfloat16 (nearest even), returned as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def random_weights(cfg, seed):
    """Random weights for a configuration (bfloat16 values held as float32), sized so that the activations stay of order one,
    the experts' clamps take part and every mechanism has a visible share of the output.  Which experts a token takes must
    not hang on rounding: the first channels (one per expert) carry a pattern of the token's own that no sublayer writes to,
    and the routers read mostly those."""
    rng = np.random.default_rng(seed)
    W, V = cfg["width"], cfg["vocab"]
    w = {}

    def lin(name, n_out, n_in, gain=1.0):
        w[name] = rng.standard_normal((n_out, n_in)) * (gain / np.sqrt(n_in))

    def vec(name, n, lo, hi):
        w[name] = rng.uniform(lo, hi, n)

    w["embed"] = 0.4 * rng.standard_normal((V, W))     # also the head: small, or every token would predict itself
    moes = [l["mlp"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"]
    R = max((m["router"]["experts"] for m in moes), default=0)
    if R:   # ranks of the experts per token, in clear steps
        order = np.argsort(rng.standard_normal((V, R)), axis=1)
        w["embed"][:, :R] = 1.5 - 3.0 * order / max(R - 1, 1)
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        H, d, r, e = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
        vec(p + "norm1", W, -0.4, 0.4)
        vec(p + "ls1", W, 0.5, 1.1)
        w[p + "ls1"][:R] = 0
        lin(p + "mix.dq", m["q_rank"], W)
        lin(p + "mix.dkv", m["kv_rank"] + r, W)
        w[p + "mix.dkv"][m["kv_rank"]:] *= 1.5
        vec(p + "mix.dq.norm", m["q_rank"], 0.6, 1.4)
        vec(p + "mix.dkv.norm", m["kv_rank"], 0.6, 1.4)
        lin(p + "mix.uq", H * (d + r), m["q_rank"], 1.5)
        lin(p + "mix.uk", H * d, m["kv_rank"], 1.5)
        lin(p + "mix.uv", H * e, m["kv_rank"], 1.5)
        vec(p + "mix.sink", H, -1.0, 2.5)
        lin(p + "mix.o", W, H * e, 1.5)
        if mlp is None:
            continue
        q = p + "mlp."
        vec(p + "norm2", W, -0.4, 0.4)
        w[p + "norm2"][:R] = 0
        vec(p + "ls2", W, 0.5, 1.1)
        w[p + "ls2"][:R] = 0
        if mlp["kind"] == "dense":
            F = mlp["ff"]
            lin(q + "gate", F, W); lin(q + "up", F, W); lin(q + "down", W, F, 1.5)
            continue
        E = mlp["router"]["experts"]
        lin(q + "router", E, W, 0.015)
        w[q + "router"][:, :R] = 2.0 * np.eye(E, R)
        parts = [(f"e{n}.", mlp["expert"]["ff"]) for n in range(E)]
        if mlp.get("shared"):
            parts.append(("shared.", mlp["shared"]["ff"]))
            lin(q + "shared.sg", 1, W)
        for n, F in parts:
            lin(q + n + "gate", F, W, 1.5); lin(q + n + "up", F, W, 1.5); lin(q + n + "down", W, F)
    vec("final.norm", W, -0.4, 0.4)
    w["final.norm"][:R] = -1
    return {k: to_bf16(v) for k, v in w.items()}
