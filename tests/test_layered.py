"""Layer-list models without a GPU: configuration, tensor names, loader and registry, the plain implementation's own
mechanisms against independent formulas, the trace replayer's order of calls, refusals of the C ABI."""
import importlib
import importlib.machinery
import importlib.util
import json
import os

import numpy as np
import pytest

from layered_common import CONFIGS, ROOT, lay, make_tensors, oracle, ref, row_errors

loader = importlib.import_module("bit-ttt-engine_b200.loader")


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_config_round_trip(name):
    cfg = CONFIGS[name]
    assert lay.gufotar_config(json.loads(json.dumps(lay.gufotar_dict(cfg)))) == cfg


def test_config_refuses_what_it_does_not_know():
    d = lay.gufotar_dict(CONFIGS["odd"])
    for edit, text in ((lambda x: x["layers"][0].update(type="other"), "mixer type"),
                       (lambda x: x["layers"][1]["mlp"].update(kind="routed"), "feed-forward kind"),
                       (lambda x: x["layers"][1]["mixer"].pop("scale"), "scale"),
                       (lambda x: x.pop("width"), "width")):
        bad = json.loads(json.dumps(d))
        edit(bad)
        with pytest.raises(loader.CheckpointError, match=text):
            lay.gufotar_config(bad)


def write_checkpoint(path, cfg, tensors):
    loader.write_safetensors(os.path.join(path, "model.safetensors"), tensors)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(lay.gufotar_dict(cfg), f)


def test_registry_chooses_the_class_by_config(tmp_path, monkeypatch):
    cfg = CONFIGS["plain"]
    t = make_tensors(cfg)
    write_checkpoint(tmp_path, cfg, t)
    seen = {}
    monkeypatch.setattr(lay, "build_layered", lambda c, tensors, **kw: seen.update(cfg=c, tensors=tensors, kw=kw) or "built")
    assert loader.load_model(str(tmp_path), max_batch=3, dtype="float32", max_seq_len=40) == "built"
    assert seen["cfg"] == cfg and seen["kw"] == {"max_batch": 3, "device": 0, "dtype": "float32", "max_seq_len": 40}
    assert all(np.array_equal(seen["tensors"][k], v) for k, v in t.items()) and seen["tensors"]["l1.mix.vmix"].shape == ()
    d = json.load(open(tmp_path / "config.json"))
    d["architecture"] = "Nothing"
    json.dump(d, open(tmp_path / "config.json", "w"))
    with pytest.raises(loader.CheckpointError, match="unknown architecture"):
        loader.load_model(str(tmp_path))


def test_missing_and_misshapen_tensors():
    cfg = CONFIGS["odd"]
    t = make_tensors(cfg)
    for name in ("l1.mix.sink", "pos", "l0.mix.conv.b", "l3.mix.vmix"):
        with pytest.raises(loader.CheckpointError, match=name):
            lay.build_layered(cfg, {k: v for k, v in t.items() if k != name})
    with pytest.raises(loader.CheckpointError, match="l0.mix.in"):
        lay.build_layered(cfg, {**t, "l0.mix.in": t["l0.mix.in"][1:]})


# ---- the plain implementation against formulas written another way --------------------

def test_sink_softmax_is_a_softmax_with_one_more_score():
    rng = np.random.default_rng(0)
    s = rng.normal(0, 3, (5, 9))
    e = np.exp(np.concatenate([s, np.full((5, 1), 1.7)], 1))
    assert np.allclose(ref.sink_softmax(s, 1.7), (e / e.sum(1, keepdims=True))[:, :9])


def test_query_temperature_steps():
    f = ref.query_temperature(np.arange(12), 0.5, 4)
    assert np.allclose(f[:3], 1.0) and np.allclose(f[3:7], 1 + 0.5 * np.log(2)) and np.allclose(f[7:11], 1 + 0.5 * np.log(3))
    assert f[11] > f[10]


def test_conv_equals_numpy_convolve():
    rng = np.random.default_rng(1)
    x, w, b = rng.normal(size=(30, 3)), rng.normal(size=(3, 4)), rng.normal(size=3)
    got = ref.causal_conv(x, w, b)
    for c in range(3):
        assert np.allclose(got[:, c], np.convolve(x[:, c], w[c, ::-1])[:30] + b[c])


def test_scan_equals_its_closed_form():
    rng = np.random.default_rng(2)
    t, h, p, g, n = 20, 4, 3, 2, 5
    x, b, c = rng.normal(size=(t, h, p)), rng.normal(size=(t, g, n)), rng.normal(size=(t, g, n))
    dt, a, d = rng.uniform(0, 1, (t, h)), rng.normal(size=h), rng.normal(size=h)
    y = ref.ssm_scan(x, b, c, dt, a, d)
    for i in (0, 7, 19):
        for k in range(h):
            want = d[k] * x[i, k]
            for j in range(i + 1):
                decay = np.exp(-np.exp(a[k]) * dt[j + 1:i + 1, k].sum())
                want = want + decay * dt[j, k] * (b[j, k // 2] @ c[i, k // 2]) * x[j, k]
            assert np.allclose(y[i, k], want)


def test_grouped_norm_and_stable_functions():
    rng = np.random.default_rng(3)
    x, w = rng.normal(size=(4, 12)), rng.normal(size=12)
    got = ref.grouped_rms_norm(x, w, 3, 1e-3)
    for g in range(3):
        s = slice(4 * g, 4 * g + 4)
        assert np.allclose(got[:, s], ref.rms_norm(x[:, s], w[s], 1e-3))
    assert np.allclose(ref.softplus(np.array([-50.0, 0.0, 50.0])), [np.exp(-50.0), np.log(2), 50.0])
    assert np.allclose(ref.relu_squared(np.array([-2.0, 3.0])), [0, 9])


def test_every_planted_flaw_changes_the_plain_logits():
    cfg = CONFIGS["odd"]
    t = make_tensors(cfg, seed=5)
    tokens = np.random.default_rng(1).integers(0, cfg.vocab_size, 40)
    base, _ = oracle(cfg, t, tokens)
    for flaw in ("no_sink", "no_cap", "no_temperature", "no_value_mix", "plain_norm", "first_key_lost", "own_key_lost", "state_lost"):
        assert row_errors(oracle(cfg, t, tokens, flaw)[0], base).max() > 0.02, flaw


# ---- trace replayer ---------------------------------------------------------------------

class FakeModel:
    def __init__(self):
        self.calls, self.current_pos = [], 0

    def reset_kv_cache(self):
        self.calls.append("reset")
        self.current_pos = 0

    def forward_one(self, tokens, want_logits=True):
        self.calls.append(("one", list(tokens), want_logits))
        self.current_pos += 1
        return np.full((1, 4), float(tokens[0]), np.float32), None

    def prefill_logits(self, tokens, want):
        self.calls.append(("prefill", list(tokens), list(want)))
        self.current_pos += len(tokens)
        return np.stack([np.full(4, float(tokens[w]), np.float32) for w in want]) if len(want) else np.zeros((0, 4), np.float32)


def load_trace_run():
    path = os.path.join(ROOT, "bin", "trace_run")
    ldr = importlib.machinery.SourceFileLoader("trace_run", path)
    mod = importlib.util.module_from_spec(importlib.util.spec_from_loader("trace_run", ldr))
    ldr.exec_module(mod)
    return mod


def test_replayer_drives_prefill_decode_and_reset():
    tr = load_trace_run()
    m = FakeModel()
    r = tr.Replayer(m)
    out = r.step([{"id": "a", "tokens": [5, 6, 7], "want": [0, 2]}], [])
    assert out.shape == (2, 4) and out[:, 0].tolist() == [5, 7]
    assert r.step([{"id": "a", "tokens": [8], "want": []}], []) is None
    assert r.step([{"id": "a", "tokens": [9], "want": [0]}], ["a"])[0, 0] == 9
    assert r.step([{"id": "b", "tokens": [1], "want": [0]}], ["b"])[0, 0] == 1  # a first token alone is a prefill
    assert m.calls == ["reset", ("prefill", [5, 6, 7], [0, 2]), ("one", [8], False), ("one", [9], True), "reset",
                       "reset", ("prefill", [1], [0]), "reset"]
    r.step([{"id": "c", "tokens": [1, 2]}], [])
    with pytest.raises(tr.TraceError):
        r.step([{"id": "d", "tokens": [1]}], [])
    with pytest.raises(tr.TraceError):
        r.step([{"id": "c", "tokens": [1], "want": [1]}], [])


def test_create_refuses_bad_layers():
    bt = importlib.import_module("bit-ttt-engine_b200")
    bt.build.build_library()
    base = CONFIGS["plain"]

    def create(**kw):
        import copy
        cfg = copy.deepcopy(base)
        for k, v in kw.items():
            setattr(cfg.layers[1], k, v)
        return bt.LayeredLM(cfg)

    for kw, text in (({"heads": 4}, "KV heads"), ({"vdim": 300}, "value heads"), ({"dim": 300}, "value heads"), ({"mixer": 7}, "unknown mixer"), ({"ff": 0}, "feed-forward"),
                     ({"vdim": 64}, "value mixing"), ({"q_temp_every": 0.0}, "q_temp_every")):
        with pytest.raises(bt.BitTTTError, match=text):
            create(**kw)
    with pytest.raises(bt.BitTTTError, match="norm groups"):
        import copy
        cfg = copy.deepcopy(base)
        cfg.layers[2].state = 300
        bt.LayeredLM(cfg)
