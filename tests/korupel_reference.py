"""Plain, slow restatement of the Korupel decoder in numpy float64: one function per mechanism, whole sequences, no
cache.  Test infrastructure; it shares no code with the library.

Weights are a dict name -> array; names and the meaning of the configuration are those of the model folder a user
loads (config.json + model.safetensors).
"""
import numpy as np


def f64(a):
    return np.asarray(a, np.float64)


def rms_norm(x, w, eps):
    x = f64(x)
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * f64(w)


def causal_conv(h, w):
    """Per channel: y[t] = sum_j w[:, j] h[t - (taps - 1) + j], zeros ahead of the sequence."""
    h, w = f64(h), f64(w)
    taps = w.shape[1]
    y = np.zeros_like(h)
    for j in range(taps):
        back = taps - 1 - j
        y[back:] += w[:, j] * h[:h.shape[0] - back] if back < h.shape[0] else 0.0
    return y


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-f64(z)))


def silu(z):
    return f64(z) * sigmoid(z)


def gelu_tanh(z):
    z = f64(z)
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def attention(q, k, r1, r2, gate, scale, size, keep_first):
    """q [T, H, d], k [T, G, d] (also the values), gate [T, H] before the sigmoid -> [T, H, d]."""
    q, k, r1, r2 = f64(q), f64(k), f64(r1), f64(r2)
    T, H, d = q.shape
    G = k.shape[1]
    pos = np.arange(T)
    dist = pos[:, None] - pos[None, :]
    mask = (dist >= 0) & ((dist < size) | (pos[None, :] < keep_first))
    out = np.zeros_like(q)
    for h in range(H):
        kv = k[:, h // (H // G)]
        s = q[:, h] @ kv.T * scale - r1[h] * np.log1p(r2[h] * np.maximum(dist, 0))
        s = np.where(mask, s, -np.inf)
        p = np.exp(s - s.max(-1, keepdims=True))
        out[:, h] = (p / p.sum(-1, keepdims=True)) @ kv
    return out * sigmoid(gate)[:, :, None]


def lightning(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, e]; S_t = decay S_{t-1} + k_t v_t^T, o_t = S_t^T q_t.  Returns (o [T, H, e], S)."""
    q, k, v, decay = f64(q), f64(k), f64(v), f64(decay)
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2])) if state is None else f64(state).copy()
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hd,hde->he", q[t], S)
    return o, S


def gated_norm(o, g, w, eps):
    """RMS norm over the concatenated heads, times sigmoid(g)."""
    return rms_norm(o, w, eps) * sigmoid(g)


def dense_ff(h, gate, up, down, act):
    return (act(h @ f64(gate).T) * (h @ f64(up).T)) @ f64(down).T


def route(h, router, top):
    """Scores sigmoid(W h) and, per token, the indices of the `top` largest."""
    s = sigmoid(h @ f64(router).T)
    return s, np.argsort(-s, axis=-1, kind="stable")[:, :top]


def moe_ff(h, w, pre, experts, top):
    s, sel = route(h, w[pre + "router"], top)
    y = np.zeros((h.shape[0], f64(w[pre + "e0.down"]).shape[0]))
    for e in range(experts):
        rows = np.nonzero((sel == e).any(-1))[0]
        if rows.size:
            y[rows] += s[rows, e][:, None] * dense_ff(h[rows], w[f"{pre}e{e}.gate"], w[f"{pre}e{e}.up"],
                                                      w[f"{pre}e{e}.down"], silu)
    return y


def mixer(h, layer, w, pre, eps):
    m, T = layer["mixer"], h.shape[0]
    if layer["type"] == "attention":
        q = h @ f64(w[pre + "q"]).T + f64(w[pre + "q.b"])
        k = h @ f64(w[pre + "k"]).T + f64(w[pre + "k.b"])
        o = attention(q.reshape(T, m["heads"], m["dim"]), k.reshape(T, m["kv_heads"], m["dim"]), w[pre + "r1"],
                      w[pre + "r2"], h @ f64(w[pre + "g"]).T, m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
        return o.reshape(T, -1) @ f64(w[pre + "o"]).T
    q, k, v = (silu(h @ f64(w[pre + n]).T).reshape(T, m["heads"], -1) for n in "qkv")
    o, _ = lightning(q, k, v, m["decay"])
    return gated_norm(o.reshape(T, -1), h @ f64(w[pre + "g"]).T, w[pre + "norm"], eps) @ f64(w[pre + "o"]).T


def feed_forward(h, layer, w, pre):
    if layer["mlp"]["kind"] == "dense":
        return dense_ff(h, w[pre + "gate"], w[pre + "up"], w[pre + "down"], gelu_tanh)
    r = layer["mlp"]["router"]
    return moe_ff(h, w, pre, r["experts"], r["top"])


def forward(cfg, w, tokens, want_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer)."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = f64(w["embed"])[np.asarray(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = rms_norm(x, w[p + "norm1"], eps)
        h = h + causal_conv(h, w[p + "canon1"])
        x = x + m * rms_norm(mixer(h, layer, w, p + "mix.", eps), w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            h = h + causal_conv(h, w[p + "canon2"])
            x = x + m * rms_norm(feed_forward(h, layer, w, p + "mlp."), w[p + "norm2b"], eps)
        streams.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ f64(w["head"]).T
    return (logits, np.stack(streams)) if want_layers else logits


# ---------------------------------------------------------------- synthetic models for the tests

def to_bf16(a):
    """Round to bfloat16 (nearest even), returned as float32."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32)


def random_weights(cfg, seed):
    """Random weights for a configuration (bfloat16 values held as float32), sized so that the activations stay of
    order one and every mechanism has a visible share of the output.  Which experts a token takes must not hang on
    rounding: the first channels (one per expert) carry a pattern of the token's own that no sublayer writes to, and the
    routers read mostly those."""
    rng = np.random.default_rng(seed)
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    w = {}

    def lin(name, n_out, n_in, gain=1.0):
        w[name] = rng.standard_normal((n_out, n_in)) * (gain / np.sqrt(n_in))

    def vec(name, n, lo, hi):
        w[name] = rng.uniform(lo, hi, n)

    w["embed"] = rng.standard_normal((V, W))
    routers = [l["mlp"]["router"] for l in cfg["layers"] if l["mlp"] and l["mlp"]["kind"] == "moe"]
    R = max((r["experts"] for r in routers), default=0)
    if R:   # ranks of the experts per token, in clear steps
        order = np.argsort(rng.standard_normal((V, R)), axis=1)
        w["embed"][:, :R] = 1.5 - 3.0 * order / max(R - 1, 1)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] is not None else ()):
            vec(p + n, W, 0.6, 1.4)
        for n in ("canon1",) + (("canon2",) if layer["mlp"] is not None else ()):
            w[p + n] = rng.standard_normal((W, taps)) * 0.4
            w[p + n][:R] = 0
        for n in ("norm1b",) + (("norm2b",) if layer["mlp"] is not None else ()):
            w[p + n][:R] = 0
        if layer["mlp"] is not None:
            w[p + "norm2"][:R] = 1
        H, d = m["heads"], m["dim"]
        if layer["type"] == "attention":
            G = m["kv_heads"]
            lin(p + "mix.q", H * d, W, 1.5)
            lin(p + "mix.k", G * d, W, 1.5)
            w[p + "mix.q.b"], w[p + "mix.k.b"] = rng.standard_normal(H * d) * 0.3, rng.standard_normal(G * d) * 0.3
            vec(p + "mix.r1", H, 0.1, 0.9)
            vec(p + "mix.r2", H, 0.05, 0.8)
            lin(p + "mix.g", H, W)
            lin(p + "mix.o", W, H * d)
        else:
            e = m["vdim"]
            lin(p + "mix.q", H * d, W)
            lin(p + "mix.k", H * d, W)
            lin(p + "mix.v", H * e, W)
            lin(p + "mix.g", H * e, W)
            lin(p + "mix.o", W, H * e)
            vec(p + "mix.norm", H * e, 0.6, 1.4)
        if layer["mlp"] is None:
            continue
        q = p + "mlp."
        if layer["mlp"]["kind"] == "dense":
            F = layer["mlp"]["ff"]
            lin(q + "gate", F, W); lin(q + "up", F, W); lin(q + "down", W, F)
        else:
            F, E = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["experts"]
            lin(q + "router", E, W, 0.015)
            w[q + "router"][:, :R] = 2.0 * np.eye(E, R)
            for e in range(E):
                lin(f"{q}e{e}.gate", F, W); lin(f"{q}e{e}.up", F, W); lin(f"{q}e{e}.down", W, F)
    vec("final.norm", W, 0.6, 1.4)
    lin("head", V, W)
    return {k: to_bf16(v) for k, v in w.items()}
