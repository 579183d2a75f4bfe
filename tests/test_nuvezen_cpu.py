"""Host side of the Nuvezen decoder: model folder reader, layer-stack description, and the plain restatement the GPU tests
compare with, checked against closed forms."""
import importlib
import math

import numpy as np
import pytest

import __graft_entry__ as entry
import nuvezen_reference as ref
import nuvezen_utils as nu


@pytest.fixture(scope="module")
def mods(pkg):
    return {n: importlib.import_module(f"{entry.PKG_NAME}.{n}") for n in ("models", "weights", "nuvezen")}


def test_norms():
    x, w = np.array([[3.0, -4.0]]), np.array([0.5, -0.25])
    r = math.sqrt(12.5 + 0.1)
    assert np.allclose(ref.rms_norm(x, w, 0.1), [[1.5 / r, 1.0 / r]])
    assert np.allclose(ref.rms_norm_zero(x, w, 0.1), [[4.5 / r, -3.0 / r]])


def test_rotation_turns_neighbours_and_keeps_relative_angles():
    x = np.zeros((1, 6))
    x[0, 2] = 1.0            # the first of pair 1
    a = 7 * 100.0 ** (-2 / 6)
    y = ref.rotate(x, [7], 100.0)
    assert np.allclose(y[0], [0, 0, math.cos(a), math.sin(a), 0, 0])
    rng = np.random.default_rng(0)
    q, k = rng.standard_normal((1, 6)), rng.standard_normal((1, 6))
    near = ref.rotate(q, [9], 50.0) @ ref.rotate(k, [4], 50.0).T
    far = ref.rotate(q, [1009], 50.0) @ ref.rotate(k, [1004], 50.0).T
    assert np.allclose(near, far)


@pytest.mark.parametrize("size", [1, 3, 50, 0])
def test_latent_attention_pair_by_pair(size):
    cfg = nu.config(24, 20, [nu.layer(2, 5, 4, 3, 7, 6, size, None, scale=0.7, base=30.0)])
    w, m = ref.random_weights(cfg, 3), cfg["layers"][0]["mixer"]
    rng = np.random.default_rng(1)
    cq, c, kr = rng.standard_normal((9, 7)), rng.standard_normal((9, 6)), rng.standard_normal((9, 4))
    out = ref.latent_attention(cq, c, kr, w, "l0.mix.", m)
    W = {n: ref.f64(w["l0.mix." + n]) for n in ("uq", "uk", "uv", "sink")}
    for i in range(9):
        for h in range(2):
            q = W["uq"][h * 9:(h + 1) * 9] @ cq[i]
            qr = ref.rotate(q[None, 5:], [i], 30.0)[0]
            num, den = np.zeros(3), math.exp(W["sink"][h])
            for j in range(i + 1):
                if size and i - j >= size:
                    continue
                s = q[:5] @ (W["uk"][h * 5:h * 5 + 5] @ c[j]) + qr @ ref.rotate(kr[j:j + 1], [j], 30.0)[0]
                e = math.exp(0.7 * s)
                num, den = num + e * (W["uv"][h * 3:h * 3 + 3] @ c[j]), den + e
            assert np.allclose(out[i, h * 3:h * 3 + 3], num / den)


def test_clamped_gate():
    eye = np.eye(1)
    for g, u in ((0.3, 0.2), (5.0, 0.2), (-5.0, 0.2), (0.3, 7.0), (0.3, -7.0)):
        gc, uc = min(g, 1.25), max(-1.25, min(u, 1.25))
        want = gc / (1 + math.exp(-1.702 * gc)) * (uc + 1)
        got = ref.clamped_ff(np.array([[1.0]]), g * eye, u * eye, eye, 1.25)
        assert np.allclose(got, want)


def test_router_takes_the_largest_logits_and_a_softmax_over_them():
    rng = np.random.default_rng(3)
    h, w = rng.standard_normal((5, 7)), rng.standard_normal((6, 7))
    sel, p = ref.route(h, w, 3)
    for t in range(5):
        z = w @ h[t]
        order = np.argsort(-z)[:3]
        assert list(sel[t]) == list(order)
        assert np.allclose(p[t], np.exp(z[order]) / np.exp(z[order]).sum())


def test_shared_expert_and_weighted_sum():
    cfg = nu.config(16, 20, [nu.layer(1, 4, 2, 4, 5, 6, 3, nu.moe(3, 2, 8, shared=12))])
    w = ref.random_weights(cfg, 5)
    h, mlp, p = np.random.default_rng(6).standard_normal((4, 16)), cfg["layers"][0]["mlp"], "l0.mlp."
    y = ref.moe_ff(h, mlp, w, p)
    sel, pr = ref.route(h, w[p + "router"], 2)
    for t in range(4):
        want = sum(pr[t, k] * ref.clamped_ff(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"], 1.5)
                   for k, e in enumerate(sel[t]))
        gate = 1 / (1 + math.exp(-float(ref.f64(w[p + "shared.sg"])[0] @ h[t])))
        want = want + gate * ref.clamped_ff(h[t], w[p + "shared.gate"], w[p + "shared.up"], w[p + "shared.down"], 0.8)
        assert np.allclose(y[t], want)


def test_both_sublayers_read_the_same_row():
    cfg = nu.config(16, 20, [nu.layer(1, 4, 2, 4, 5, 6, 3, nu.dense(8))])
    w = ref.random_weights(cfg, 5)
    x, l = np.random.default_rng(7).standard_normal((4, 16)), cfg["layers"][0]
    a = ref.mixer(ref.rms_norm_zero(x, w["l0.norm1"], 0.2), l["mixer"], w, "l0.mix.", 0.2)
    f = ref.feed_forward(ref.rms_norm_zero(x, w["l0.norm2"], 0.2), l["mlp"], w, "l0.mlp.")
    assert np.allclose(ref.layer_step(x, l, w, "l0.", 0.2), x + ref.f64(w["l0.ls1"]) * a + ref.f64(w["l0.ls2"]) * f)


# ------------------------------------------------------------------------------ what the library is given

@pytest.mark.parametrize("name", sorted(nu.CONFIGS))
def test_layer_description(mods, name):
    cfg, w = nu.make(name)
    M = mods["models"]
    layers = mods["nuvezen"].stack_layers(cfg, {k: nu.bits(v) for k, v in w.items()}.__getitem__)
    assert len(layers) == len(cfg["layers"])
    for i, (d, l) in enumerate(zip(layers, cfg["layers"])):
        m, mlp = l["mixer"], l["mlp"]
        H, R = m["heads"], m["kv_rank"]
        assert d["form"] == M.LAYER_PARALLEL and d["mixer"] == M.MIXER_LATENT_ATTENTION and d["window"] == m["mask"]["size"]
        assert d["w_in"].shape == ((m["q_rank"] + R + m["rot_dim"] + 7) // 8 * 8, cfg["width"])
        assert d["w_ukv"].shape == (H * (m["dim"] + m["vdim"]), R) and d["w_ukt"].shape == (H, R, m["dim"])
        uk = nu.bits(w[f"l{ref.owner(cfg, i)}.mix.uk"])
        assert (d["w_ukt"][H - 1].T == uk[(H - 1) * m["dim"]:]).all() and (d["w_ukv"][:H * m["dim"]] == uk).all()
        if l.get("weights_of") is not None:     # the same arrays, so that they are uploaded once
            assert d is layers[l["weights_of"]]
        assert (d["ff"] == M.FF_NONE) == (mlp is None)
        if mlp and mlp["kind"] == "moe":
            E = mlp["router"]["experts"]
            assert d["w_gate_up"].shape[0] == E and d["router"].shape[0] == E + (1 if mlp.get("shared") else 0)
            assert d["router_kind"] == M.ROUTER_SOFTMAX and d["act"] == M.ACT_CLAMPED and d["act_limit"] == mlp["expert"]["limit"]


def test_weights_of_chains_and_circles(mods):
    N = mods["nuvezen"]
    assert N.owner([{}, {"weights_of": 0}, {"weights_of": 1}], 2) == 0
    with pytest.raises(ValueError, match="circle"):
        N.owner([{"weights_of": 1}, {"weights_of": 0}], 0)


def test_wrong_sizes_are_reported(mods):
    cfg, w = nu.make("even")
    get = {k: nu.bits(v) for k, v in w.items()}
    bad = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], vdim=16))])
    with pytest.raises(ValueError, match="uv"):
        mods["nuvezen"].stack_layers(bad, get.__getitem__)
    bad = dict(cfg, layers=[dict(cfg["layers"][0], mixer=dict(cfg["layers"][0]["mixer"], rot={"base": 10.0, "dims": 4}))])
    with pytest.raises(ValueError, match="rot"):
        mods["nuvezen"].stack_layers(bad, get.__getitem__)
    with pytest.raises(ValueError, match="mixer"):
        mods["nuvezen"].stack_layers(dict(cfg, layers=[dict(cfg["layers"][0], type="other")]), get.__getitem__)


def test_registry_names_the_design(mods, tmp_path):
    (tmp_path / "config.json").write_text('{"architecture": "Unheard"}')
    with pytest.raises(ValueError, match="Nuvezen"):
        mods["models"].load_model(None, str(tmp_path))


def test_norm_weights_become_factors(mods):
    w = ref.to_bf16(np.array([0.5, -0.25, 0.0, -1.0]))
    assert (mods["nuvezen"].norm_weight(nu.bits(w)) == np.array([1.5, 0.75, 1.0, 0.0], np.float32)).all()
