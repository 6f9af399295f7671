"""The layer-list design `Fepapel` without a GPU: configuration, tensor names, registry, refusals, and the plain
implementation's mechanisms against formulas written another way."""
import copy
import importlib
import json

import numpy as np
import pytest

from fepapel_common import CONFIGS, FLAWS, lay, latent, make_tensors, oracle, ref, rglru, row_errors, wkv

loader = importlib.import_module("bit-ttt-engine_b200.loader")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_round_trip(name):
    cfg = CONFIGS[name]
    assert lay.fepapel_config(json.loads(json.dumps(lay.fepapel_dict(cfg))), make_tensors(cfg)) == cfg


def test_config_refuses_what_it_does_not_know():
    cfg = CONFIGS["loop"]
    d, t = lay.fepapel_dict(cfg), make_tensors(cfg)
    for edit, text in ((lambda x: x["layers"][0].update(type="mamba2"), "mixer type"),
                       (lambda x: x["layers"][0]["mlp"].update(kind="dense"), "feed-forward kind"),
                       (lambda x: x["layers"][1]["mixer"].pop("rot"), "rot"),
                       (lambda x: x["layers"][1]["mixer"]["rot"].pop("base"), "base"),
                       (lambda x: x["loop"].pop("times"), "times"), (lambda x: x.pop("norm"), "norm")):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(loader.CheckpointError, match=text):
            lay.fepapel_config(bad, t)
    with pytest.raises(loader.CheckpointError, match="l2.mix.w1"):
        lay.fepapel_config(d, {k: v for k, v in t.items() if k != "l2.mix.w1"})


def test_registry_and_tensor_names(tmp_path, monkeypatch):
    cfg = CONFIGS["odd"]
    t = make_tensors(cfg)
    loader.write_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(lay.fepapel_dict(cfg)))
    seen = {}
    monkeypatch.setattr(lay, "build_layered", lambda c, tensors, **kw: seen.update(cfg=c, tensors=tensors) or "built")
    assert loader.load_model(str(tmp_path), dtype="float32") == "built"
    assert seen["cfg"] == cfg and seen["cfg"].layers[0].decay_rank == 5  # a size that only the tensors tell
    names = [n for n, _, _, _ in lay.tensor_shapes(cfg)]
    assert len(set(names)) == len(names) == len(t)
    for name in ("loop.in", "loop.step", "l0.norm1b", "l0.mix.mu.w", "l1.mix.dkv.norm", "l1.mlp.e6.down", "l2.mix.ra.b", "l2.mlp.shared.up"):
        assert name in names
    monkeypatch.undo()
    for name in ("l1.mix.g", "l2.mlp.e2.up", "loop.step", "l0.norm2b"):
        with pytest.raises(loader.CheckpointError, match=name):
            lay.build_layered(cfg, {k: v for k, v in t.items() if k != name})
    with pytest.raises(loader.CheckpointError, match="l0.mlp.router"):
        lay.build_layered(cfg, {**t, "l0.mlp.router": t["l0.mlp.router"][1:]})


def test_layer_runs():
    assert CONFIGS["loop"].runs() == [0, 1, 2, 1, 2, 1, 2, 3]
    assert CONFIGS["odd"].runs() == [0, 1, 2, 0, 1, 2] and CONFIGS["wide"].runs() == [0, 1, 2, 3]
    for cfg in CONFIGS.values():
        assert [i for i, _ in ref.layer_runs(lay.fepapel_dict(cfg))] == cfg.runs()
    assert [t for _, t in ref.layer_runs(lay.fepapel_dict(CONFIGS["loop"]))] == [None, 0, None, 1, None, 2, None, None]


# ---- the plain implementation against formulas written another way --------------------

def test_rotation_is_a_complex_product():
    rng = np.random.default_rng(0)
    x, pos = rng.normal(size=(5, 3, 10)), np.array([0, 1, 7, 100, 5000])
    got = ref.rotate_pairs(x, pos, 300.0, 6)
    z = (x[..., 0:6:2] + 1j * x[..., 1:6:2]) * np.exp(1j * pos[:, None, None] * 300.0 ** (-np.arange(3) / 3.0))
    assert np.allclose(got[..., 0:6:2], z.real) and np.allclose(got[..., 1:6:2], z.imag) and np.array_equal(got[..., 6:], x[..., 6:])


def test_wkv_scan_equals_its_closed_form():
    rng = np.random.default_rng(1)
    t, h, d = 12, 2, 5
    r, k, v, u = rng.normal(size=(t, h, d)), rng.normal(size=(t, h, d)), rng.normal(size=(t, h, d)), rng.normal(size=(h, d))
    w = rng.uniform(0, 1, (t, h, d))
    o = ref.wkv_scan(r, k, v, w, u)
    for i in (0, 1, 11):
        for a in range(h):
            want = (r[i, a] * u[a]) @ k[i, a] * v[i, a]
            for j in range(i):
                want = want + (r[i, a] * w[j + 1:i, a].prod(0)) @ k[j, a] * v[j, a]
            assert np.allclose(o[i, a], want)


def test_gated_linear_recurrence_equals_its_closed_form():
    rng = np.random.default_rng(2)
    u, r, i, lam = rng.normal(size=(9, 4)), rng.uniform(size=(9, 4)), rng.uniform(size=(9, 4)), rng.normal(size=4)
    a = np.exp(-8 * r * np.log1p(np.exp(lam)))
    s = ref.rglru_scan(u, r, i, lam)
    for t in (0, 3, 8):
        assert np.allclose(s[t], sum(a[j + 1:t + 1].prod(0) * np.sqrt(1 - a[j] ** 2) * i[j] * u[j] for j in range(t + 1)))


def test_block_product_is_block_diagonal():
    rng = np.random.default_rng(3)
    w, b, x = rng.normal(size=(3, 4, 4)), rng.normal(size=(3, 4)), rng.normal(size=(6, 12))
    full = np.zeros((12, 12))
    for i in range(3):
        full[4 * i:4 * i + 4, 4 * i:4 * i + 4] = w[i]
    assert np.allclose(ref.block_product(x, w, b), x @ full.T + b.reshape(-1))


def test_attention_and_mixture_against_loops():
    rng = np.random.default_rng(4)
    q, k, v = rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 3)), rng.normal(size=(6, 2, 4))
    o = ref.causal_softmax_attention(q, k, v, 0.7)
    for i in range(6):
        e = np.exp(0.7 * (k[:i + 1, 1] @ q[i, 1]))
        assert np.allclose(o[i, 1], e @ v[:i + 1, 1] / e.sum())
    cfg = CONFIGS["loop"]
    w = ref.sub(make_tensors(cfg), "l0.mlp.", np.float64)
    h = rng.normal(size=(7, 128))
    got = ref.moe(h, w, lay.fepapel_dict(cfg)["layers"][0]["mlp"])
    z = h @ w["router"].T + w["router.b"]
    mask = z >= np.sort(z, axis=1)[:, -2:-1]
    p = np.where(mask, np.exp(z), 0)
    p /= p.sum(1, keepdims=True)
    want = ref.gated_mlp(h, w, "shared.") + sum(p[:, e:e + 1] * ref.gated_mlp(h, w, f"e{e}.") for e in range(6))
    assert mask.sum(1).tolist() == [2] * 7 and np.allclose(got, want)
    x = np.linspace(-4, 4, 41)
    assert np.allclose(ref.sigmoid(x), 1 / (1 + np.exp(-x))) and abs(ref.gelu_tanh(np.array(1.0)) - 0.841192) < 1e-5


def test_every_planted_flaw_changes_the_plain_logits():
    cfg = CONFIGS["loop"]
    t = make_tensors(cfg, seed=5)
    tokens = np.random.default_rng(1).integers(0, cfg.vocab_size, 40)
    base, _ = oracle(cfg, t, tokens)
    for flaw in FLAWS:
        assert row_errors(oracle(cfg, t, tokens, flaw)[0], base).max() > 0.01, flaw


def test_create_refuses_bad_layers():
    bt = importlib.import_module("bit-ttt-engine_b200")
    bt.build.build_library()
    for layer, kw, text in ((0, {"blocks": 7}, "blocks"), (0, {"conv_taps": 0}, "taps"), (0, {"top": 9}, "experts"), (0, {"experts": 0}, "experts"),
                            (1, {"kv_rank": 600}, "latent rank"), (1, {"rot_dims": 15}, "rotated"), (1, {"rot_dim": 200}, "rotated"),
                            (2, {"dim": 300}, "wkv heads"), (2, {"decay_rank": 0}, "decay rank"), (1, {"mixer": 9}, "unknown mixer")):
        cfg = copy.deepcopy(CONFIGS["loop"])
        for k, v in kw.items():
            setattr(cfg.layers[layer], k, v)
        with pytest.raises(bt.BitTTTError, match=text):
            bt.LayeredLM(cfg)
    for loop in ((1, 1, 2), (2, 5, 2), (-1, 2, 2)):
        cfg = copy.deepcopy(CONFIGS["loop"])
        cfg.loop = loop
        with pytest.raises(bt.BitTTTError, match="loop"):
            bt.LayeredLM(cfg)


def test_builders_cover_every_mixer():
    kinds = {c.mixer for cfg in CONFIGS.values() for c in cfg.layers}
    assert kinds == {latent(1, 1, 2, 1, 1).mixer, wkv(1, 1, 1).mixer, rglru(1, 1, 1).mixer}
