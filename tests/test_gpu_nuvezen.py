"""The Nuvezen decoder on the GPU against its plain restatement: each mechanism alone, whole prompts, portions, decoding,
batches, reuse of requests, window edges, and generation through the framework's loop."""
import importlib
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import __graft_entry__ as entry
import nuvezen_reference as ref
import nuvezen_utils as nu

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def mods(pkg):
    return {n: importlib.import_module(f"{entry.PKG_NAME}.{n}") for n in ("models", "nuvezen", "parallel")}


_reference = {}


def expected(name, n, seed=0):
    """Tokens and float64 logits of a synthetic model (computed once per module run)."""
    key = (name, n, seed)
    if key not in _reference:
        cfg, w = nu.make(name)
        toks = nu.tokens(cfg, n, seed)
        _reference[key] = (toks, ref.forward(cfg, w, toks))
    return _reference[key]


class Model:
    def __init__(self, ctx, mods, cfg, w, dtype, max_seq=512):
        self.m = mods["nuvezen"].from_tensors(ctx, cfg, {k: nu.bits(v) for k, v in w.items()}, dtype=dtype, max_seq=max_seq)

    def __enter__(self):
        return self.m

    def __exit__(self, *exc):
        self.m.close()


def model(ctx, mods, name, dtype, max_seq=512):
    return Model(ctx, mods, *nu.make(name), dtype, max_seq)


def run(m, r, toks, cuts=()):
    """Logits of toks fed in portions that end at the given places."""
    out, at = [], 0
    for end in [c for c in cuts if 0 < c < len(toks)] + [len(toks)]:
        out.append(m.step(r, toks[at:end], range(end - at))[0])
        at = end
    return np.concatenate(out)


def compare(ctx, mods, cfg, w, toks, dtype, cuts=(), what=""):
    with Model(ctx, mods, cfg, w, dtype, max_seq=len(toks)) as m:
        r = m.request()
        got = run(m, r, toks, cuts)
        r.close()
    nu.assert_logits(got, ref.forward(cfg, w, toks), dtype, what)


# ------------------------------------------------------------------------------ each mechanism alone

def small(size=9, mlp=None, dim=16):
    return nu.layer(2, dim, 8, 24, 32, 40, size, mlp)


MECHANISMS = {
    "latent attention": [nu.layer(4, 32, 16, 48, 40, 56, 20, None)],
    "latent attention, every key": [nu.layer(5, 24, 8, 16, 24, 64, 0, None)],
    "latent attention, odd sizes": [nu.layer(3, 7, 6, 5, 9, 11, 13, None, base=20.0)],
    "latent attention, one head": [nu.layer(1, 64, 32, 72, 80, 136, 33, None, scale=-0.05)],
    "latent attention, seventeen heads": [nu.layer(17, 8, 8, 8, 48, 24, 70, None)],
    "dense": [small(mlp=nu.dense(112))],
    "experts": [small(mlp=nu.moe(10, 3, 40))],
    "experts, all of them": [small(mlp=nu.moe(4, 4, 32, limit=0.5))],
    "shared expert, wider": [small(mlp=nu.moe(6, 1, 32, shared=200))],
    "shared expert, narrower": [small(mlp=nu.moe(6, 2, 136, limit=2.0, shared=16, shared_limit=0.2))],
    "weights used again": [small(mlp=nu.moe(6, 2, 40, shared=40)), nu.again([small(mlp=nu.moe(6, 2, 40, shared=40))], 0)],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 75])
@pytest.mark.parametrize("what", sorted(MECHANISMS))
def test_mechanism(ctx, mods, what, width, dtype):
    cfg = nu.config(width, 48, MECHANISMS[what])
    compare(ctx, mods, cfg, ref.random_weights(cfg, 7), nu.tokens(cfg, 150), dtype, (90, 91, 93), what)


@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_epsilon_and_weights(ctx, mods, dtype):
    """A large epsilon and weights far from zero: their share of the output cannot be missed."""
    cfg = nu.config(64, 48, [small(mlp=nu.dense(32)), small(mlp=nu.moe(4, 2, 32, shared=32))], eps=0.5)
    w = ref.random_weights(cfg, 8)
    for n in w:
        if n.endswith(("norm1", "norm2", "final.norm")):
            w[n] = ref.to_bf16(np.where(w[n] == -1, -1, w[n] * 2 + 0.7))
    for cuts in ((), (1, 2, 3), (7, 9, 11, 40)):
        compare(ctx, mods, cfg, w, nu.tokens(cfg, 45), dtype, cuts, f"cuts {cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size", [3, 60])
def test_sink(ctx, mods, size, dtype):
    """Heads whose sink takes nearly all of the weight, about half, and none."""
    cfg = nu.config(64, 48, [nu.layer(4, 16, 8, 24, 32, 40, size, None)])
    w = ref.random_weights(cfg, 9)
    w["l0.mix.sink"] = ref.to_bf16(np.array([8.0, np.log(min(size, 30)), -90.0, 60.0]))
    toks = nu.tokens(cfg, 130)
    want = ref.forward(cfg, w, toks)
    without = ref.forward(cfg, dict(w, **{"l0.mix.sink": np.full(4, -90.0)}), toks)
    assert np.median(nu.rel_err(without, want)) > 0.3, "the sinks must show"
    with Model(ctx, mods, cfg, w, dtype) as m:
        r = m.request()
        for cuts in ((), range(1, 130), (64, 66, 90)):
            r.reset()
            nu.assert_logits(run(m, r, toks, cuts), want, dtype, f"size {size}")
        r.close()


@pytest.mark.parametrize("name", ["odd", "even"])
def test_residual_stream_after_every_layer(ctx, mods, name):
    cfg, w = nu.make(name)
    toks = nu.tokens(cfg, 21)
    _, streams = ref.forward(cfg, w, toks, want_layers=True)
    with Model(ctx, mods, cfg, w, "float32") as m:
        ctx.set_option("stack_trace", 1)
        try:
            r = m.request()
            got, _ = m.step(r, toks, range(21))
            for i, want in enumerate(streams):
                assert np.abs(m.layer_stream(r, i, len(toks)) - want).max() < 1e-4 * np.abs(want).max(), i
            nu.assert_logits(got, ref.forward(cfg, w, toks), "float32", "traced")
            r.close()
        finally:
            ctx.set_option("stack_trace", 0)


# ------------------------------------------------------------------------------ prompts, portions, decoding

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(nu.CONFIGS))
def test_whole_prompts(ctx, mods, name, dtype):
    with model(ctx, mods, name, dtype) as m:
        for n in (1, 2, 8, 9, 64, 65, 129, 300):
            toks, want = expected(name, n)
            r = m.request()
            got, tok = m.step(r, toks, range(n), want_token=True)
            assert tok == int(np.argmax(got[-1]))
            nu.assert_logits(got, want, dtype, f"{name}, {n} tokens")
            r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(nu.CONFIGS))
def test_token_by_token_equals_the_prompt(ctx, mods, name, dtype):
    toks, want = expected(name, 300)
    with model(ctx, mods, name, dtype) as m:
        r = m.request()
        got = run(m, r, toks, range(150, 300))
        assert len(r) == 300
        nu.assert_logits(got, want, dtype, name)
        r.reset()
        nu.assert_logits(run(m, r, toks[:40], range(1, 40)), want[:40], dtype, f"{name} from the first token")
        r.close()


@pytest.mark.parametrize("name", ["even", "wide", "long"])
def test_both_prompt_kernels(ctx, mods, name):
    """The tcgen05 kernel and the one that takes the head sizes it cannot hold."""
    toks, want = expected(name, 300)
    try:
        for option in (1, 0):
            ctx.set_option("attn_tc", option)
            with model(ctx, mods, name, "bfloat16") as m:
                r = m.request()
                for cuts in ((), (5, 130, 133, 270)):
                    r.reset()
                    nu.assert_logits(run(m, r, toks, cuts), want, "bfloat16", f"{name}, attn_tc {option}, cuts {cuts}")
                r.close()
    finally:
        ctx.set_option("attn_tc", -1)


PORTIONS = [tuple(range(2, 300, 2)), tuple(range(3, 300, 7)), (1, 3, 66, 69, 133, 135, 136, 200, 263, 266), tuple(range(64, 300, 64)),
            tuple(range(8, 300, 9)), (299,)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(nu.CONFIGS))
def test_portions(ctx, mods, name, dtype):
    toks, want = expected(name, 300)
    with model(ctx, mods, name, dtype) as m:
        r = m.request()
        for cuts in PORTIONS:
            r.reset()
            nu.assert_logits(run(m, r, toks, cuts), want, dtype, f"{name}, portions {cuts[:6]}")
        r.close()


def test_a_repeated_prompt_is_replayed_from_a_recording(ctx, mods):
    """The third run of a shape launches a recorded graph; other shapes and another request's longer prompt (which moves the
    buffer that expanded keys share) run in between and must not disturb what it leaves."""
    toks, want = expected("even", 129)
    long_toks, long_want = expected("even", 300)
    with model(ctx, mods, "even", "bfloat16") as m:
        r, other = m.request(), m.request()
        for i in range(6):
            r.reset()
            got, _ = m.step(r, toks[:128], [0, 127])
            nu.assert_logits(got, want[[0, 127]], "bfloat16", f"run {i}")
            got, _ = m.step(r, toks[128:], [0])
            nu.assert_logits(got, want[128:], "bfloat16", f"run {i}, decoded")
            if i == 3:
                got, _ = m.step(other, long_toks, [299])
                nu.assert_logits(got, long_want[299:], "bfloat16", "the longer prompt")
        r.close()
        other.close()


def test_long_decoding(ctx, mods):
    cfg, w = nu.make("even")
    toks = nu.tokens(cfg, 700, seed=5)
    want = ref.forward(cfg, w, toks)
    with Model(ctx, mods, cfg, w, "bfloat16", max_seq=700) as m:
        r = m.request()
        nu.assert_logits(run(m, r, toks, range(60, 700)), want, "bfloat16", "640 decoded tokens")
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_decoding_through_many_tiles(ctx, mods, dtype):
    """More tiles of keys than the blocks of a cluster: every block walks several, also an unequal number of them."""
    cfg = nu.config(64, 48, [nu.layer(4, 16, 8, 24, 32, 40, 0, None), nu.layer(2, 16, 16, 16, 32, 520, 700, None)])
    w = ref.random_weights(cfg, 15)
    toks = nu.tokens(cfg, 1000)
    want = ref.forward(cfg, w, toks)
    with Model(ctx, mods, cfg, w, dtype, max_seq=1000) as m:
        r = m.request()
        cuts = [500, 501, 502, 511, 512, 513, 514, 575, 576, 577, 578, 830, 831, 832, 833, 998, 999]
        nu.assert_logits(run(m, r, toks, cuts), want, dtype, "many tiles")
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even"])
def test_requests_are_independent_and_reused(ctx, mods, name, dtype):
    """Steps of several requests in turn, and requests that end and whose memory serves the next one."""
    sets = [expected(name, n, seed) for n, seed in ((70, 1), (23, 2), (110, 3), (5, 4))]
    with model(ctx, mods, name, dtype) as m:
        pool = mods["models"].RequestPool(m)
        at, got = [0] * 4, [[] for _ in sets]
        order = np.random.default_rng(0)
        while any(a < len(t) for a, (t, _) in zip(at, sets)):
            i = int(order.integers(0, 4))
            t = sets[i][0]
            if at[i] >= len(t):
                continue
            n = min(int(order.integers(1, 12)), len(t) - at[i])
            got[i].append(m.step(pool.get(i), t[at[i]:at[i] + n], range(n))[0])
            at[i] += n
            if at[i] == len(t):
                pool.end(i)
        for i, (t, want) in enumerate(sets):
            nu.assert_logits(np.concatenate(got[i]), want, dtype, f"request {i}")
        for i, (t, want) in enumerate(sets):   # every one of these runs in memory another request has used
            assert len(pool.free) >= 1 and not pool.live
            nu.assert_logits(run(m, pool.get(("again", i)), t, (2, 9)), want, dtype, f"request {i} again")
            pool.end(("again", i))
        pool.close()


# ------------------------------------------------------------------------------ edges of windows, far keys

def needle_model(size, dim=32, rot=16, heads=4, vdim=24, q_rank=32, kv_rank=40, width=64, rotated=False):
    """One attention layer in which token 1 ('asks') gives a query that only the key of token 0 ('needle') answers, with a
    score far above all others: whether the needle is visible decides the output.  rotated: the answer lies in the shared
    rotated key part, which is turned so slowly that the distance does not matter."""
    cfg = nu.config(width, 32, [nu.layer(heads, dim, rot, vdim, q_rank, kv_rank, size, None, scale=0.5, base=1e30 if rotated else 100.0)])
    w = ref.random_weights(cfg, 11)
    rng = np.random.default_rng(12)
    w["embed"] = ref.to_bf16(np.eye(32, width) * 4 + 0.05 * w["embed"])
    p = "l0.mix."
    a, b = np.sign(rng.standard_normal(q_rank)), np.sign(rng.standard_normal(kv_rank))
    w["l0.norm1"] = np.zeros(width, np.float32)
    w[p + "dq.norm"], w[p + "dkv.norm"] = np.ones(q_rank, np.float32), np.ones(kv_rank, np.float32)
    w[p + "dq"][:, 1] = a                 # token 1's query latent is a, token 0's key latent is b
    w[p + "dkv"][:kv_rank, 0] = b
    u = np.sign(rng.standard_normal(dim)) * (28.0 / dim) ** 0.5
    uq, uk = 0.05 * w[p + "uq"].reshape(heads, dim + rot, q_rank), 0.2 * w[p + "uk"]
    w[p + "dkv"][kv_rank:] *= 0.1
    if rotated:
        v = np.zeros(rot)
        v[2:] = np.sign(rng.standard_normal(rot - 2))     # (pair 0 turns with the position itself)
        uq[:, dim:] = np.outer(v * 3.0, a) / q_rank
        w[p + "dkv"][kv_rank:, 0] = v / 4
    else:
        uq[:, :dim] += np.outer(u, a) / q_rank
        uk += np.tile(np.outer(u, b) / kv_rank, (heads, 1))
    w[p + "uq"], w[p + "uk"] = uq.reshape(-1, q_rank), uk
    w[p + "o"] = w[p + "o"] * 3
    return cfg, {k: ref.to_bf16(v) for k, v in w.items()}


def needle_tokens(n, needle, asks, seed=3):
    t = np.random.default_rng(seed).integers(2, 32, n)
    t[needle], t[asks] = 0, 1
    return t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,rot,heads,rotated", [(32, 16, 4, False), (64, 64, 18, True), (30, 6, 2, False), (8, 32, 3, True)])
@pytest.mark.parametrize("size", [1, 2, 17, 64, 65, 100])
def test_window_edge(ctx, mods, size, dim, rot, heads, rotated, dtype):
    """A needle just inside and just outside the window, in a prompt and decoded."""
    cfg, w = needle_model(size, dim, rot, heads, rotated=rotated)
    n = 210
    with Model(ctx, mods, cfg, w, dtype, max_seq=n) as m:
        r = m.request()
        for asks in (size + 2, 131, 191, n - 1):
            seen = []
            for needle in (asks - size + 1, asks - size):
                if needle == asks:      # a window of one: the query sees itself only
                    continue
                t = needle_tokens(n, needle, asks)
                want = ref.forward(cfg, w, t)
                seen.append(want[asks])
                for cuts in ((), (asks, asks + 1), (asks - 1, asks + 2)):
                    r.reset()
                    nu.assert_logits(run(m, r, t, cuts)[asks:asks + 1], want[asks:asks + 1], dtype, f"size {size} needle {needle} asks {asks} cuts {cuts}")
            if len(seen) == 2:
                assert nu.rel_err(seen[0][None], seen[1][None])[0] > 0.3, "the needle must show"
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rotated", [False, True])
def test_far_keys_through_an_unlimited_window(ctx, mods, rotated, dtype):
    cfg, w = needle_model(0, rotated=rotated)
    n = 520
    with Model(ctx, mods, cfg, w, dtype, max_seq=n) as m:
        r = m.request()
        for needle, asks in ((0, n - 1), (63, 500), (64, 511), (255, 513), (450, 519)):
            t = needle_tokens(n, needle, asks)
            want = ref.forward(cfg, w, t)
            other = t.copy()
            other[needle] = 5
            assert nu.rel_err(ref.forward(cfg, w, other)[asks:asks + 1], want[asks:asks + 1])[0] > 0.3, "the needle must show"
            for cuts in ((), (asks, asks + 1), (256,)):
                r.reset()
                nu.assert_logits(run(m, r, t, cuts)[asks:asks + 1], want[asks:asks + 1], dtype, f"needle {needle} asks {asks}")
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_rotation_far_from_the_start(ctx, mods, dtype):
    """Scores made of the rotated part alone, with pairs that turn fast and slowly, a thousand tokens in."""
    cfg = nu.config(64, 48, [nu.layer(2, 8, 32, 24, 32, 40, 40, None, scale=0.4, base=200.0)])
    w = ref.random_weights(cfg, 16)
    uq = w["l0.mix.uq"].reshape(2, 40, 32)
    uq[:, :8] = 0
    w["l0.mix.sink"][:] = -3
    toks = nu.tokens(cfg, 1100)
    want = ref.forward(cfg, w, toks)
    with Model(ctx, mods, cfg, w, dtype, max_seq=1100) as m:
        r = m.request()
        nu.assert_logits(run(m, r, toks, (1000, 1003, 1004, 1005)), want, dtype, "rotation")
        r.close()


# ------------------------------------------------------------------------------ generation and serving

def greedy_ok(cfg, w, prompt, toks, dtype):
    """Every generated token is the restatement's choice for the sequence so far wherever that choice is clear."""
    seq = np.concatenate([prompt, toks])
    lo = ref.forward(cfg, w, seq[:-1])[len(prompt) - 1:]
    spread = np.sqrt(((lo - lo.mean(-1, keepdims=True)) ** 2).mean())
    margin = {"float32": 1e-3, "bfloat16": 0.15}[dtype] * spread
    clear = 0
    for row, tok in zip(lo, toks):
        top = np.sort(row)[-2:]
        if top[1] - top[0] > margin:
            clear += 1
            assert int(np.argmax(row)) == int(tok)
    assert clear > len(toks) // 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even", "wide"])
def test_greedy_generation(ctx, mods, name, dtype):
    cfg, w = nu.make(name)
    with Model(ctx, mods, cfg, w, dtype) as m:
        r, r2 = m.request(), m.request()
        prompt = nu.tokens(cfg, 37, seed=9)
        _, first = m.step(r, prompt, want_token=True)
        toks, logits = m.generate(r, first, 24, want_logits=True)
        assert logits.shape == (24, cfg["vocab"]) and logits.dtype == np.float32
        greedy_ok(cfg, w, prompt, np.concatenate([[first], toks]), dtype)
        assert len(r) == 37 + 24
        # the step entry point fed with the same tokens gives the same logits
        m.step(r2, prompt)
        seq = np.concatenate([[first], toks[:-1]])
        got = np.concatenate([m.step(r2, [t], [0])[0] for t in seq])
        nu.assert_logits(logits, got.astype(np.float64), dtype, "generate against step")
        # teacher forcing follows the given tokens
        forced = nu.tokens(cfg, 10, seed=10).astype(np.uint32)
        r.reset()
        m.step(r, prompt)
        _, logits = m.generate(r, forced[0], 9, forced=forced[1:], want_logits=True)
        want = ref.forward(cfg, w, np.concatenate([prompt, forced[:9]]))[37:]
        nu.assert_logits(logits, want, dtype, "forced")
        r.close()
        r2.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even", "wide", "long"])
def test_batched_generation_equals_single(ctx, mods, name, dtype):
    """Up to eight requests of unequal lengths in one step, each against itself alone."""
    cfg, w = nu.make(name)
    lens = [40, 1, 77, 8, 130, 2, 64, 33]
    with Model(ctx, mods, cfg, w, dtype) as m:
        forced = np.stack([nu.tokens(cfg, 12, seed=30 + i) for i in range(8)]).astype(np.uint32)
        reqs = [m.request() for _ in lens]
        for n in (2, 3, 8):
            firsts = []
            for i in range(n):
                reqs[i].reset()
                firsts.append(m.step(reqs[i], nu.tokens(cfg, lens[i], seed=20 + i), want_token=True)[1])
            toks = m.generate_batch(reqs[:n], firsts, 12, forced=forced[:n])
            for i in range(n):
                # what the batch left in the request: the next token's logits against the restatement
                seq = np.concatenate([nu.tokens(cfg, lens[i], seed=20 + i), [firsts[i]], forced[i][:11]])
                want = ref.forward(cfg, w, np.concatenate([seq, forced[i][11:]]))
                got, _ = m.step(reqs[i], forced[i][11:], [0])
                assert len(reqs[i]) == lens[i] + 13
                nu.assert_logits(got, want[-1:], dtype, f"{name}: request {i} of {n}")
                lo = want[lens[i]:lens[i] + 12]
                gap = np.sort(lo, -1)
                clear = gap[:, -1] - gap[:, -2] > 0.3 * lo.std()
                assert (toks[i][clear] == lo.argmax(-1)[clear]).mean() > (0.999 if dtype == "float32" else 0.8) if clear.any() else True
        for r in reqs:
            r.close()


def test_serving_prompts_without_images(ctx, mods):
    cfg, w = nu.make("even")
    with Model(ctx, mods, cfg, w, "bfloat16") as m:
        par = mods["parallel"]
        requests = [par.Request(None, nu.tokens(cfg, n, seed=n)) for n in (5, 61, 17, 128, 9)]
        out = par.serve_requests(ctx, None, m, requests, 1, 0, 10, max_streams=3)
        for i, rq in enumerate(requests):
            assert out[i].shape == (11,)
            greedy_ok(cfg, w, rq.ids, out[i], "bfloat16")


def test_errors(ctx, mods, pkg):
    with model(ctx, mods, "ones", "float32", max_seq=8) as m:
        r = m.request()
        with pytest.raises(pkg.MdError) as e:
            m.step(r, np.zeros(9))
        assert e.value.status == 4          # MD_ERR_SEQUENCE_TOO_LONG
        with pytest.raises(pkg.MdError):
            m.step(r, [m.vocab])
        assert len(r) == 0
        r.close()
    cfg, w = nu.make("even")
    layers = mods["nuvezen"].stack_layers(cfg, {k: nu.bits(v) for k, v in w.items()}.__getitem__)
    kw = dict(embed=w["embed"], head=None, final_norm=w["final.norm"], eps=1e-5)
    for change in (dict(form=mods["models"].LAYER_SANDWICH), dict(router_kind=7), dict(kv_rank=40), dict(q_norm=None), dict(act=9), dict(sink=None)):
        with pytest.raises(pkg.MdError):
            mods["models"].StackModel(ctx, [dict(layers[0], **change)], **kw)


# ------------------------------------------------------------------------------ the command line programs

@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(tmp_path, dtype):
    cfg, w = nu.make("odd")
    (tmp_path / "model").mkdir()
    (tmp_path / "out").mkdir()
    nu.write_folder(tmp_path / "model", cfg, w)
    (ta, wa), (tb, wb) = expected("odd", 70, 1), expected("odd", 23, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:50].tolist(), "want": [0, 7, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": ta[50:69].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": tb.tolist(), "want": [22]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": ta[69:].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "a", "tokens": tb[:3].tolist(), "want": [0, 1, 2]}], "end": ["a"]}]
    p = subprocess.run([os.path.join(entry.ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype, "--out",
                        str(tmp_path / "out"), "--max-tokens", "100"], input="".join(json.dumps(s) + "\n" for s in steps),
                       text=True, capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr
    assert p.stdout.split("\n")[:5] == [f"done {i}" for i in range(5)]

    def got(i):
        return np.fromfile(tmp_path / "out" / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])
    assert not (tmp_path / "out" / "1.f32").exists()
    nu.assert_logits(np.concatenate([got(0), got(3)]), wa[[0, 7, 49, 69]], dtype)
    nu.assert_logits(np.concatenate([got(2), got(4)]), wb[[22, 0, 1, 2]], dtype)


def test_generate_program(tmp_path):
    cfg, w = nu.make("even")
    nu.write_folder(tmp_path, cfg, w)
    prompts = [nu.tokens(cfg, n, seed=n) for n in (12, 30)]
    p = subprocess.run([sys.executable, os.path.join(entry.ROOT, "bin", "generate"), "--model", str(tmp_path), "--steps", "16"] +
                       sum([["--tokens", ",".join(map(str, t))] for t in prompts], []), text=True, capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr
    lines = [np.array([int(x) for x in ln.split()]) for ln in p.stdout.strip().split("\n")]
    assert [ln.size for ln in lines] == [16, 16]
    for t, ln in zip(prompts, lines):
        greedy_ok(cfg, w, t, ln, "bfloat16")
