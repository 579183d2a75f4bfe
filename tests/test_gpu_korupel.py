"""The Korupel decoder on the GPU against its plain restatement: each mechanism alone, whole prompts, portions, decoding,
batches, reuse of requests, window edges, and generation through the framework's loop."""
import importlib
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import __graft_entry__ as entry
import korupel_reference as ref
import korupel_utils as ku

pytestmark = pytest.mark.gpu
DTYPES = ["float32", "bfloat16"]


@pytest.fixture(scope="module")
def mods(pkg):
    return {n: importlib.import_module(f"{entry.PKG_NAME}.{n}") for n in ("models", "korupel", "parallel")}


_reference = {}


def expected(name, n, seed=0):
    """Tokens and float64 logits of a synthetic model (computed once per module run)."""
    key = (name, n, seed)
    if key not in _reference:
        cfg, w = ku.make(name)
        toks = ku.tokens(cfg, n, seed)
        _reference[key] = (toks, ref.forward(cfg, w, toks))
    return _reference[key]


class Model:
    def __init__(self, ctx, mods, cfg, w, dtype, max_seq=512):
        self.m = mods["korupel"].from_tensors(ctx, cfg, {k: ku.bits(v) for k, v in w.items()}, dtype=dtype, max_seq=max_seq)

    def __enter__(self):
        return self.m

    def __exit__(self, *exc):
        self.m.close()


def model(ctx, mods, name, dtype, max_seq=512):
    return Model(ctx, mods, *ku.make(name), dtype, max_seq)


def run(m, r, toks, cuts=(), start=0):
    """Logits of toks[start:] fed in portions that end at the given places."""
    out, at = [], start
    for end in [c for c in cuts if start < c < len(toks)] + [len(toks)]:
        out.append(m.step(r, toks[at:end], range(end - at))[0])
        at = end
    return np.concatenate(out)


def compare(ctx, mods, cfg, w, toks, dtype, cuts=(), what=""):
    with Model(ctx, mods, cfg, w, dtype, max_seq=len(toks)) as m:
        r = m.request()
        got = run(m, r, toks, cuts)
        r.close()
    ku.assert_logits(got, ref.forward(cfg, w, toks), dtype, what)


# ------------------------------------------------------------------------------ each mechanism alone

MECHANISMS = {
    "attention": [ku.attention(4, 2, 48, 20, 3, None)],
    "attention, every key": [ku.attention(5, 5, 24, 1000, 0, None)],
    "attention, one key head": [ku.attention(12, 1, 16, 11, 4, None)],
    "lightning": [ku.lightning(3, 40, 56, None)],
    "lightning, decay 1": [ku.lightning(2, 64, 64, None, decay=[1.0, 1.0])],
    "lightning, fast decay": [ku.lightning(3, 16, 24, None, decay=[1e-4, 0.03, 0.3])],
    "dense": [ku.lightning(1, 8, 8, ku.dense(112))],
    "experts": [ku.lightning(1, 8, 8, ku.moe(10, 3, 40))],
    "experts, all of them": [ku.lightning(1, 8, 8, ku.moe(4, 4, 32))],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [64, 75])
@pytest.mark.parametrize("what", sorted(MECHANISMS))
def test_mechanism(ctx, mods, what, width, dtype):
    cfg = ku.config(width, 48, 3, MECHANISMS[what])
    w = ref.random_weights(cfg, 7)
    compare(ctx, mods, cfg, w, ku.tokens(cfg, 150), dtype, (90, 91, 93), what)


@pytest.mark.parametrize("taps", [1, 2, 3, 5])
def test_convolution_and_norms(ctx, mods, taps):
    """Strong convolution weights and a large epsilon: their share of the output cannot be missed."""
    cfg = ku.config(64, 48, taps, [ku.lightning(1, 8, 8, ku.dense(32)), ku.attention(2, 1, 16, 4, 1, ku.dense(32))], eps=0.3)
    w = ref.random_weights(cfg, 8)
    for n in list(w):
        if "canon" in n:
            w[n] = ref.to_bf16(w[n] * 3)
    for cuts in ((), (1, 2, 3), (7, 9, 11, 40)):
        compare(ctx, mods, cfg, w, ku.tokens(cfg, 45), "float32", cuts, f"{taps} taps, cuts {cuts}")


def test_residual_stream_after_every_layer(ctx, mods):
    cfg, w = ku.make("odd")
    toks = ku.tokens(cfg, 21)
    _, streams = ref.forward(cfg, w, toks, want_layers=True)
    with Model(ctx, mods, cfg, w, "float32") as m:
        ctx.set_option("stack_trace", 1)
        try:
            r = m.request()
            m.step(r, toks)
            for i, want in enumerate(streams):
                assert np.abs(m.layer_stream(r, i, len(toks)) - want).max() < 1e-4 * np.abs(want).max(), i
            r.close()
        finally:
            ctx.set_option("stack_trace", 0)


# ------------------------------------------------------------------------------ prompts, portions, decoding

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ku.CONFIGS))
def test_whole_prompts(ctx, mods, name, dtype):
    with model(ctx, mods, name, dtype) as m:
        for n in (1, 2, 9, 64, 65, 129, 300):
            toks, want = expected(name, n)
            r = m.request()
            got, tok = m.step(r, toks, range(n), want_token=True)
            assert tok == int(np.argmax(got[-1]))
            ku.assert_logits(got, want, dtype, f"{name}, {n} tokens")
            r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ku.CONFIGS))
def test_token_by_token_equals_the_prompt(ctx, mods, name, dtype):
    toks, want = expected(name, 300)
    with model(ctx, mods, name, dtype) as m:
        r = m.request()
        got = run(m, r, toks, range(150, 300))
        assert len(r) == 300
        ku.assert_logits(got, want, dtype, name)
        r.reset()
        ku.assert_logits(run(m, r, toks[:40], range(1, 40)), want[:40], dtype, f"{name} from the first token")
        r.close()


PORTIONS = [tuple(range(2, 300, 2)), tuple(range(3, 300, 7)), (1, 3, 66, 69, 133, 135, 136, 200, 263, 266), tuple(range(64, 300, 64)),
            tuple(range(8, 300, 9)), (299,)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(ku.CONFIGS))
def test_portions(ctx, mods, name, dtype):
    toks, want = expected(name, 300)
    with model(ctx, mods, name, dtype) as m:
        r = m.request()
        for cuts in PORTIONS:
            r.reset()
            ku.assert_logits(run(m, r, toks, cuts), want, dtype, f"{name}, portions {cuts[:6]}")
        r.close()


def test_a_repeated_prompt_is_replayed_from_a_recording(ctx, mods):
    """The third run of a shape launches a recorded graph; other shapes run in between must not disturb what it leaves."""
    toks, want = expected("even", 129)
    with model(ctx, mods, "even", "bfloat16") as m:
        r = m.request()
        for i in range(4):
            r.reset()
            got, _ = m.step(r, toks[:128], [0, 127])
            ku.assert_logits(got, want[[0, 127]], "bfloat16", f"run {i}")
            got, _ = m.step(r, toks[128:], [0])
            ku.assert_logits(got, want[128:], "bfloat16", f"run {i}, decoded")
        r.close()


def test_long_decoding(ctx, mods):
    cfg, w = ku.make("even")
    toks = ku.tokens(cfg, 700, seed=5)
    want = ref.forward(cfg, w, toks)
    with Model(ctx, mods, cfg, w, "bfloat16", max_seq=700) as m:
        r = m.request()
        ku.assert_logits(run(m, r, toks, range(60, 700)), want, "bfloat16", "640 decoded tokens")
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_requests_are_independent_and_reused(ctx, mods, dtype):
    """Steps of several requests in turn, and requests that end and whose memory serves the next one."""
    sets = [expected("odd", n, seed) for n, seed in ((70, 1), (23, 2), (110, 3), (5, 4))]
    with model(ctx, mods, "odd", dtype) as m:
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
            ku.assert_logits(np.concatenate(got[i]), want, dtype, f"request {i}")
        for i, (t, want) in enumerate(sets):   # every one of these runs in memory another request has used
            assert len(pool.free) >= 1 and not pool.live
            ku.assert_logits(run(m, pool.get(("again", i)), t, (2, 9)), want, dtype, f"request {i} again")
            pool.end(("again", i))
        pool.close()


# ------------------------------------------------------------------------------ edges of windows, far keys

def needle_model(size, keep, dim=32, heads=4, kv_heads=2, width=64, layers=1):
    """Attention layers in which token 1 ('asks') gives a query that only the key of token 0 ('needle') answers, with a
    score far above all others: whether the needle is visible decides the output."""
    cfg = ku.config(width, 32, 2, [ku.attention(heads, kv_heads, dim, size, keep, None, scale=0.5) for _ in range(layers)], mult=1.0)
    w = ref.random_weights(cfg, 11)
    w["embed"] = ref.to_bf16(np.eye(32, width) * 8 + 0.05 * w["embed"])
    for i in range(layers):
        p = f"l{i}."
        w[p + "canon1"] = np.zeros_like(w[p + "canon1"])
        for n in ("norm1", "norm1b"):
            w[p + n] = np.ones_like(w[p + n])
        u = np.sign(np.random.default_rng(12).standard_normal(dim)) * 0.4
        q, k = 0.05 * w[p + "mix.q"], 0.3 * w[p + "mix.k"]
        q[:, 1] = np.tile(u, heads)
        k[:, 0] = np.tile(u, kv_heads)
        w[p + "mix.q"], w[p + "mix.k"] = ref.to_bf16(q), ref.to_bf16(k)
        w[p + "mix.q.b"], w[p + "mix.k.b"] = 0 * w[p + "mix.q.b"], 0 * w[p + "mix.k.b"]
        w[p + "mix.r1"], w[p + "mix.r2"] = ref.to_bf16(0.5 * w[p + "mix.r1"]), w[p + "mix.r2"]
    return cfg, w


def needle_tokens(n, needle, asks, seed=3):
    t = np.random.default_rng(seed).integers(2, 32, n)
    t[needle], t[asks] = 0, 1
    return t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,heads,kv_heads", [(32, 4, 2), (64, 8, 1), (36, 2, 2)])
@pytest.mark.parametrize("size", [1, 2, 17, 64, 65, 100])
def test_window_edge(ctx, mods, size, dim, heads, kv_heads, dtype):
    """A needle just inside and just outside the window, in a prompt and decoded."""
    cfg, w = needle_model(size, 0, dim, heads, kv_heads)
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
                    ku.assert_logits(run(m, r, t, cuts)[asks:asks + 1], want[asks:asks + 1], dtype, f"size {size} needle {needle} asks {asks} cuts {cuts}")
            if len(seen) == 2:
                assert ku.rel_err(seen[0][None], seen[1][None])[0] > 0.3, "the needle must show"
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("keep", [0, 1, 3, 20])
def test_first_tokens_are_kept(ctx, mods, keep, dtype):
    cfg, w = needle_model(9, keep)
    n = 150
    with Model(ctx, mods, cfg, w, dtype, max_seq=n) as m:
        r = m.request()
        for needle in sorted({0, max(keep - 1, 0), keep, keep + 1}):
            for asks in (needle + 5, needle + 30, 128, n - 1):
                t = needle_tokens(n, needle, asks)
                want = ref.forward(cfg, w, t)
                for cuts in ((), (asks, asks + 1), (asks - 3, asks + 4)):
                    r.reset()
                    ku.assert_logits(run(m, r, t, cuts)[asks:asks + 1], want[asks:asks + 1], dtype, f"keep {keep} needle {needle} asks {asks} cuts {cuts}")
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_keys_through_an_unlimited_window(ctx, mods, dtype):
    cfg, w = needle_model(4096, 0)
    n = 520
    with Model(ctx, mods, cfg, w, dtype, max_seq=n) as m:
        r = m.request()
        for needle, asks in ((0, n - 1), (63, 500), (64, 511), (255, 513), (450, 519)):
            t = needle_tokens(n, needle, asks)
            want = ref.forward(cfg, w, t)
            for cuts in ((), (asks, asks + 1), (256,)):
                r.reset()
                ku.assert_logits(run(m, r, t, cuts)[asks:asks + 1], want[asks:asks + 1], dtype, f"needle {needle} asks {asks}")
        r.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_pulse_in_the_recurrence(ctx, mods, dtype):
    """One token writes a key ten times the others' size; with a decay near one it must still show far behind, whatever
    the portions."""
    cfg = ku.config(64, 48, 2, [ku.lightning(2, 32, 32, None, decay=[0.9999, 0.9995])])
    w = ref.random_weights(cfg, 13)
    w["embed"][:, 0] = 0
    w["embed"][0] = 0
    w["embed"][0, 0] = 8            # a channel no other token has: k is large there, v as ever
    w["l0.canon1"][0] = 0
    w["l0.mix.k"][:, 0] = 40
    w["l0.mix.v"][:, 0] = ref.to_bf16(np.sign(w["l0.mix.v"][:, 0]))
    w["l0.mix.q"] = ref.to_bf16(w["l0.mix.q"] * 2)
    t = np.random.default_rng(14).integers(1, 48, 400)
    t[3] = 0
    want = ref.forward(cfg, w, t)
    other = t.copy()
    other[3] = 1
    assert ku.rel_err(want[-20:], ref.forward(cfg, w, other)[-20:]).min() > 0.2, "the pulse must show"
    with Model(ctx, mods, cfg, w, dtype) as m:
        r = m.request()
        for cuts in ((), (2, 5), (64, 128, 192, 256), tuple(range(380, 400))):
            r.reset()
            ku.assert_logits(run(m, r, t, cuts), want, dtype, f"cuts {cuts[:4]}")
        r.close()


# ------------------------------------------------------------------------------ generation and serving

def greedy_ok(cfg, w, prompt, toks, dtype):
    """Every generated token is the restatement's choice for the sequence so far wherever that choice is clear."""
    seq = np.concatenate([prompt, toks])
    lo = ref.forward(cfg, w, seq[:-1])[len(prompt) - 1:]
    spread = np.sqrt(((lo - lo.mean(-1, keepdims=True)) ** 2).mean())
    margin = {"float32": 1e-3, "bfloat16": 0.25}[dtype] * spread
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
    cfg, w = ku.make(name)
    with Model(ctx, mods, cfg, w, dtype) as m:
        r, r2 = m.request(), m.request()
        prompt = ku.tokens(cfg, 37, seed=9)
        _, first = m.step(r, prompt, want_token=True)
        toks, logits = m.generate(r, first, 24, want_logits=True)
        assert logits.shape == (24, cfg["vocab"]) and logits.dtype == np.float32
        greedy_ok(cfg, w, prompt, np.concatenate([[first], toks]), dtype)
        assert len(r) == 37 + 24
        # the step entry point fed with the same tokens gives the same logits
        m.step(r2, prompt)
        seq = np.concatenate([[first], toks[:-1]])
        got = np.concatenate([m.step(r2, [t], [0])[0] for t in seq])
        ku.assert_logits(logits, got.astype(np.float64), dtype, "generate against step")
        # teacher forcing follows the given tokens
        forced = ku.tokens(cfg, 10, seed=10).astype(np.uint32)
        r.reset()
        m.step(r, prompt)
        _, logits = m.generate(r, forced[0], 9, forced=forced[1:], want_logits=True)
        want = ref.forward(cfg, w, np.concatenate([prompt, forced[:9]]))[37:]
        ku.assert_logits(logits, want, dtype, "forced")
        r.close()
        r2.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["odd", "even", "wide"])
def test_batched_generation_equals_single(ctx, mods, name, dtype):
    """Up to eight requests of unequal lengths in one step, each against itself alone."""
    cfg, w = ku.make(name)
    lens = [40, 1, 77, 8, 130, 2, 64, 33]
    with Model(ctx, mods, cfg, w, dtype) as m:
        forced = np.stack([ku.tokens(cfg, 12, seed=30 + i) for i in range(8)]).astype(np.uint32)
        reqs = [m.request() for _ in lens]
        for n in (2, 3, 8):
            firsts = []
            for i in range(n):
                reqs[i].reset()
                firsts.append(m.step(reqs[i], ku.tokens(cfg, lens[i], seed=20 + i), want_token=True)[1])
            toks = m.generate_batch(reqs[:n], firsts, 12, forced=forced[:n])
            for i in range(n):
                # what the batch left in the request: the next token's logits against the restatement
                seq = np.concatenate([ku.tokens(cfg, lens[i], seed=20 + i), [firsts[i]], forced[i][:11]])
                want = ref.forward(cfg, w, np.concatenate([seq, forced[i][11:]]))
                got, _ = m.step(reqs[i], forced[i][11:], [0])
                assert len(reqs[i]) == lens[i] + 13
                ku.assert_logits(got, want[-1:], dtype, f"{name}: request {i} of {n}")
                lo = want[lens[i]:lens[i] + 12]
                gap = np.sort(lo, -1)
                clear = gap[:, -1] - gap[:, -2] > 0.3 * lo.std()
                assert (toks[i][clear] == lo.argmax(-1)[clear]).mean() > (0.999 if dtype == "float32" else 0.8)
        for r in reqs:
            r.close()


def test_serving_prompts_without_images(ctx, mods):
    cfg, w = ku.make("even")
    with Model(ctx, mods, cfg, w, "bfloat16") as m:
        par = mods["parallel"]
        requests = [par.Request(None, ku.tokens(cfg, n, seed=n)) for n in (5, 61, 17, 128, 9)]
        out = par.serve_requests(ctx, None, m, requests, 1, 0, 10, max_streams=3)
        for i, rq in enumerate(requests):
            assert out[i].shape == (11,)
            greedy_ok(cfg, w, rq.ids, out[i], "bfloat16")


def test_the_phi_decoder_takes_the_same_step(ctx, mods):
    """md_text_step on the older text model: same logits as embedding + forward."""
    from model_utils import text_weights
    w = text_weights(3, n_layers=2, dim=128, hidden=256, vocab=96)
    m = mods["models"].TextModel(ctx, w, n_heads=2, max_seq=64)
    a, b = m.request(), m.request()
    ids = np.array([5, 17, 90, 2, 33, 8, 1, 70, 44, 21], np.uint32)
    _, want, tok = m.forward(a, m.text_encoder(ids))
    got, tok2 = m.step(b, ids, [3, 9], want_token=True)
    assert tok == tok2 and np.array_equal(got[1], want.astype(np.float32)) and len(b) == 10
    _, want, _ = m.forward(a, m.text_encoder([7]))
    got, _ = m.step(b, [7], [0])
    assert np.array_equal(got[0], want.astype(np.float32))
    for r in (a, b):
        r.close()
    m.close()


def test_errors(ctx, mods, pkg):
    with model(ctx, mods, "ones", "float32", max_seq=8) as m:
        r = m.request()
        with pytest.raises(pkg.MdError) as e:
            m.step(r, np.zeros(9))
        assert e.value.status == 4          # MD_ERR_SEQUENCE_TOO_LONG
        with pytest.raises(pkg.MdError):
            m.step(r, [m.vocab])
        with pytest.raises(pkg.MdError):
            m.step(r, [1, 2], [2])
        with pytest.raises(pkg.MdError):
            m.text_encoder([1])
        assert len(r) == 0
        m.step(r, [1, 2, 3])
        with pytest.raises(pkg.MdError):
            m.generate(r, 0, 6)
        r.close()


# ------------------------------------------------------------------------------ the command line programs

@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(tmp_path, dtype):
    cfg, w = ku.make("odd")
    (tmp_path / "model").mkdir()
    (tmp_path / "out").mkdir()
    ku.write_folder(tmp_path / "model", cfg, w)
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
    ku.assert_logits(np.concatenate([got(0), got(3)]), wa[[0, 7, 49, 69]], dtype)
    ku.assert_logits(np.concatenate([got(2), got(4)]), wb[[22, 0, 1, 2]], dtype)


def test_generate_program(tmp_path):
    cfg, w = ku.make("even")
    ku.write_folder(tmp_path, cfg, w)
    prompts = [ku.tokens(cfg, n, seed=n) for n in (12, 30)]
    p = subprocess.run([sys.executable, os.path.join(entry.ROOT, "bin", "generate"), "--model", str(tmp_path), "--steps", "8"] +
                       sum([["--tokens", ",".join(map(str, t))] for t in prompts], []), text=True, capture_output=True, timeout=600)
    assert p.returncode == 0, p.stderr
    lines = [np.array([int(x) for x in ln.split()]) for ln in p.stdout.strip().split("\n")]
    assert [ln.size for ln in lines] == [8, 8]
    for t, ln in zip(prompts, lines):
        greedy_ok(cfg, w, t, ln, "bfloat16")
