"""Small synthetic Nuvezen models for the tests: configurations of deliberately odd and of kernel-friendly sizes."""
import nuvezen_reference as ref
from korupel_utils import assert_logits, bits, rel_err, tokens, write_folder  # noqa: F401  (the designs share these helpers)


def layer(heads, dim, rot, vdim, q_rank, kv_rank, size, mlp, scale=None, base=10000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": scale or (dim + rot) ** -0.5, "mask": {"size": size}, "rot": {"base": base, "dims": rot}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit=1.5, shared=None, shared_limit=0.8):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared, "limit": shared_limit}
    return m


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Nuvezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


def again(layers, j):
    """A layer that runs layer j's weights."""
    return dict(layers[j], weights_of=j)


def _odd():
    l = [layer(3, 10, 6, 14, 22, 18, 7, moe(5, 2, 24, shared=40)), layer(5, 9, 2, 7, 13, 30, 23, dense(50), base=50.0)]
    return l + [again(l, 1), again(l, 0), layer(2, 12, 4, 5, 17, 11, 0, None), layer(4, 6, 8, 20, 33, 40, 5, moe(4, 4, 11, limit=0.6))]


def _even():
    l = [layer(6, 32, 8, 24, 56, 72, 100, moe(16, 3, 64, shared=96)), layer(8, 48, 16, 64, 128, 120, 33, dense(320), base=500.0)]
    return l + [again(l, 0), layer(2, 64, 64, 128, 64, 104, 65, moe(9, 4, 96, limit=3.0, shared=32, shared_limit=0.3)), again(l, 0)]


CONFIGS = {
    # every branch, sizes that no fast path can take whole
    "odd": config(90, 61, _odd(), eps=3e-4),
    # values that are 1 or equal: a window of one token, one head, one expert per token, latents of one value
    "ones": config(32, 40, [layer(1, 1, 2, 1, 1, 1, 1, moe(3, 1, 32, shared=32)), layer(1, 32, 32, 32, 32, 32, 2, dense(32)),
                            layer(2, 8, 2, 8, 16, 16, 3, moe(1, 1, 8)), layer(32, 1, 2, 1, 32, 32, 1, None)], eps=0.05),
    # multiples of 8: the tensor-core and vector paths
    "even": config(160, 136, _even()),
    # more heads than one block of the decode kernel takes, and not a multiple of it
    "wide": config(256, 264, [layer(20, 64, 32, 64, 192, 256, 200, moe(24, 6, 128, shared=128)), layer(40, 16, 16, 16, 96, 64, 70, dense(512))]),
    # the longest head sizes and latents of the tensor-core kernels
    "long": config(128, 72, [layer(3, 128, 64, 128, 136, 512, 150, dense(64)), layer(2, 208, 48, 200, 88, 648, 90, None)]),
}


def make(name, seed=1):
    cfg = CONFIGS[name]
    return cfg, ref.random_weights(cfg, seed)
