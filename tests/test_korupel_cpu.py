"""Host side of the Korupel decoder: model folder reader, layer-stack description, and the plain restatement the GPU
tests compare with, checked against closed forms."""
import importlib

import numpy as np
import pytest

import __graft_entry__ as entry
import korupel_reference as ref
import korupel_utils as ku


@pytest.fixture(scope="module")
def mods(pkg):
    return {n: importlib.import_module(f"{entry.PKG_NAME}.{n}") for n in ("models", "weights", "korupel")}


def test_causal_conv_is_a_shifted_sum():
    rng = np.random.default_rng(0)
    h, w = rng.standard_normal((6, 3)), rng.standard_normal((3, 4))
    y = ref.causal_conv(h, w)
    for t in range(6):
        for c in range(3):
            want = sum(w[c, j] * h[t - 3 + j, c] for j in range(4) if t - 3 + j >= 0)
            assert abs(y[t, c] - want) < 1e-12


def test_lightning_recurrence_equals_its_closed_form():
    rng = np.random.default_rng(1)
    q, k, v = rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 3)), rng.standard_normal((9, 2, 5))
    decay = np.array([0.7, 1.0])
    o, S = ref.lightning(q, k, v, decay)
    for t in range(9):
        for h in range(2):
            want = sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1))
            assert np.allclose(o[t, h], want)
    o2, S2 = ref.lightning(q[4:], k[4:], v[4:], decay, ref.lightning(q[:4], k[:4], v[:4], decay)[1])
    assert np.allclose(o2, o[4:]) and np.allclose(S2, S)


@pytest.mark.parametrize("size,keep", [(1, 0), (3, 0), (3, 2), (2, 5), (50, 0)])
def test_attention_mask_and_bias(size, keep):
    rng = np.random.default_rng(2)
    q, k, gate = rng.standard_normal((8, 4, 6)), rng.standard_normal((8, 2, 6)), rng.standard_normal((8, 4))
    r1, r2 = rng.uniform(0.1, 1, 4), rng.uniform(0.1, 1, 4)
    out = ref.attention(q, k, r1, r2, gate, 0.4, size, keep)
    for i in range(8):
        for h in range(4):
            js = [j for j in range(i + 1) if ref.visible(i, j, size, keep)]
            s = np.array([q[i, h] @ k[j, h // 2] * 0.4 - r1[h] * np.log(1 + r2[h] * (i - j)) for j in js])
            p = np.exp(s - s.max())
            want = (p / p.sum()) @ k[js, h // 2] / (1 + np.exp(-gate[i, h]))
            assert np.allclose(out[i, h], want)


def test_router_takes_the_largest_scores_unnormalised():
    rng = np.random.default_rng(3)
    h, w = rng.standard_normal((5, 7)), rng.standard_normal((6, 7))
    s, sel = ref.route(h, w, 2)
    for t in range(5):
        order = sorted(range(6), key=lambda e: -(h[t] @ w[e]))
        assert list(sel[t]) == order[:2]
        assert np.allclose(s[t], 1 / (1 + np.exp(-(w @ h[t]))))


def test_gate_up_blocks_and_padding(mods):
    k = mods["korupel"]
    gate, up = np.arange(40 * 3).reshape(40, 3), 1000 + np.arange(40 * 3).reshape(40, 3)
    gu = k.gate_up(gate, up)
    assert gu.shape == (128, 3)
    for j in range(64):
        row = (j // 32) * 64 + j % 32
        assert (gu[row] == (gate[j] if j < 40 else 0)).all()
        assert (gu[row + 32] == (up[j] if j < 40 else 0)).all()
    d = k.down(np.arange(2 * 40).reshape(2, 40))
    assert d.shape == (2, 64) and (d[:, 40:] == 0).all() and (d[:, :40] == np.arange(80).reshape(2, 40)).all()


@pytest.mark.parametrize("name", sorted(ku.CONFIGS))
def test_layer_description(mods, name):
    cfg, w = ku.make(name)
    layers = mods["korupel"].stack_layers(cfg, {k: ku.bits(v) for k, v in w.items()}.__getitem__)
    assert len(layers) == len(cfg["layers"])
    for d, layer in zip(layers, cfg["layers"]):
        m = layer["mixer"]
        rows = ((m["heads"] + m["kv_heads"]) * m["dim"] + m["heads"] if layer["type"] == "attention"
                else 2 * m["heads"] * (m["dim"] + m["vdim"]))
        assert d["w_in"].shape == ((rows + 7) // 8 * 8, cfg["width"])
        assert d["w_out"].shape == (cfg["width"], m["heads"] * m["vdim"])
        assert (d["ff"] == mods["models"].FF_NONE) == (layer["mlp"] is None)
        if layer["mlp"] and layer["mlp"]["kind"] == "moe":
            assert d["w_gate_up"].shape[0] == layer["mlp"]["router"]["experts"] == d["experts"]


def test_safetensors_reader(mods, tmp_path):
    cfg, w = ku.make("ones")
    ku.write_folder(tmp_path, cfg, w)
    with mods["weights"].SafetensorsFile(str(tmp_path / "model.safetensors")) as t:
        assert set(t.keys()) == set(w)
        for n, a in w.items():
            assert t[n].shape == a.shape and (mods["models"].StackModel.widen(t[n]) == a).all()
        with pytest.raises(KeyError):
            t["absent"]
    raw = (tmp_path / "model.safetensors").read_bytes()
    (tmp_path / "cut").write_bytes(raw[:len(raw) - 10])
    with mods["weights"].SafetensorsFile(str(tmp_path / "cut")) as t:
        with pytest.raises(ValueError):
            t[list(w)[-1]]
    (tmp_path / "short").write_bytes(b"\xff" * 12)
    with pytest.raises(ValueError):
        mods["weights"].SafetensorsFile(str(tmp_path / "short"))


def test_registry_names_the_design(mods, tmp_path):
    assert "Korupel" in mods["models"].MODELS
    (tmp_path / "config.json").write_text('{"architecture": "Unheard"}')
    with pytest.raises(ValueError, match="Unheard"):
        mods["models"].load_model(None, str(tmp_path))


def test_bfloat16_rounding_helpers_agree(mods):
    a = np.random.default_rng(4).standard_normal(1000).astype(np.float32)
    S = mods["models"].StackModel
    assert (S.widen(S.narrow(a)) == ref.to_bf16(a)).all()
