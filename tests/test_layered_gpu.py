"""Layer-list models on the GPU against the plain implementation (oracle/layered.py): whole prompts, portions, decoding,
batches, reuse of the caches, far keys at tile borders, each mechanism alone, sizes that fill several tiles."""
import importlib

import numpy as np
import pytest

from gpu_util import load_bt
from layered_common import A, CONFIGS, attn, bf16, lay, make_tensors, oracle, ref, row_errors, ssm

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu

# Errors relative to the root mean square of what is expected: the largest of any position, and the root mean square over
# the positions.  bf16 models multiply bf16 activations; single positions where a sublayer's output is small (its norm
# blows the rounding up) lie well above the mean.
TOL = {"float32": (3e-5, 1e-5), "bfloat16": (0.15, 0.02)}


def assert_close(got, want, dtype, what=""):
    e = row_errors(got, want)
    assert e.max() <= TOL[dtype][0] and np.sqrt((e * e).mean()) <= max(TOL[dtype][1], TOL[dtype][0] / np.sqrt(len(e))), (what, e.max(), np.sqrt((e * e).mean()))


@pytest.fixture(scope="module")
def bt():
    if not torch.cuda.is_available():
        pytest.fail("GPU tests need a CUDA device")
    mod = load_bt()
    yield mod
    assert mod.lib().bt_device_check(0) == 0


_CASES = {}


def case(name, n=90, seed=0):
    """(config, tensors, tokens, oracle logits, oracle stream), computed once."""
    key = (name, n, seed)
    if key not in _CASES:
        cfg = CONFIGS[name]
        t = make_tensors(cfg, seed=seed)
        tokens = np.random.default_rng(seed + 1).integers(0, cfg.vocab_size, n).astype(np.int32)
        _CASES[key] = (cfg, t, tokens, *oracle(cfg, t, tokens))
    return _CASES[key]


def feed(m, tokens, sizes):
    """All logits of `tokens` fed in portions (1 = decode step), sizes repeated as needed."""
    out, at, i = [], 0, 0
    while at < len(tokens):
        n = min(sizes[i % len(sizes)], len(tokens) - at)
        part = tokens[at:at + n]
        out.append(m.forward_one(part)[0] if n == 1 and at > 0 else m.prefill_logits(part, np.arange(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_whole_prompt_and_stream_after_every_layer(bt, name, dtype):
    cfg, t, tokens, logits, stream = case(name)
    m = lay.build_layered(cfg, t, dtype=dtype)
    assert_close(m.prefill_logits(tokens, np.arange(len(tokens))), logits, dtype)
    m.reset_kv_cache()
    m.set_trace(True, rows=len(tokens))
    m.prefill(tokens)
    got = m.read_trace(len(tokens))
    m.set_trace(False)
    for i in range(len(cfg.layers)):
        assert_close(got[i], stream[i], dtype, f"layer {i}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_token_by_token(bt, name, dtype):
    cfg, t, tokens, logits, stream = case(name)
    m = lay.build_layered(cfg, t, dtype=dtype)
    for sizes in ([1], [2], [3, 17, 1, 2], [31, 5], [64, 1], [16]):
        m.reset_kv_cache()
        assert_close(feed(m, tokens, sizes), logits, dtype, sizes)
    # the stream after every layer of a decode step, traced (launch by launch)
    m.reset_kv_cache()
    m.prefill(tokens[:-1])
    m.set_trace(True)
    m.forward_one(tokens[-1:])
    got = m.read_trace(1)
    m.set_trace(False)
    for i in range(len(cfg.layers)):
        scale = np.sqrt((stream[i] ** 2).mean())
        assert np.abs(got[i, 0] - stream[i, -1]).max() <= (1e-4 if dtype == "float32" else 0.15) * scale, f"layer {i}"


@pytest.mark.parametrize("flaw", ["no_sink", "no_cap", "no_temperature", "no_value_mix", "plain_norm", "first_key_lost",
                                  "own_key_lost", "state_lost"])
def test_a_planted_flaw_of_the_oracle_shows(bt, flaw):
    cfg, t, tokens, logits, _ = case("odd", 60, 3)
    m = lay.build_layered(cfg, t, dtype="float32")
    for got in (m.prefill_logits(tokens, np.arange(len(tokens))), (m.reset_kv_cache(), feed(m, tokens, [20, 1]))[1]):
        assert_close(got, logits, "float32")
        assert row_errors(got, oracle(cfg, t, tokens, flaw)[0]).max() > 100 * TOL["float32"][0]


# ---- one mechanism at a time, through the stream after a single layer ------------------------------------------------

def layer_mix(cfg, t, tokens):
    """The mixer's output of a one-layer model, from its parts: switches of the layer's configuration respected."""
    c, w = cfg.layers[0], ref.sub(t, "l0.mix.", np.float64)
    x = np.asarray(t["embed"], np.float64)[tokens] + (np.asarray(t["pos"], np.float64)[:len(tokens)] if cfg.max_positions and "pos" in t else 0)
    n, H, G = len(tokens), c.heads, c.kv_heads
    q, k, v = x @ w["q"].T, x @ w["k"].T, (x @ w["v"].T).reshape(n, G, c.vdim)
    if c.qk_norm:
        q, k = ref.rms_norm(q, w["q.norm"], cfg.norm_eps), ref.rms_norm(k, w["k.norm"], cfg.norm_eps)
    if c.q_temp_coef:
        q = q * ref.query_temperature(np.arange(n), c.q_temp_coef, c.q_temp_every)[:, None]
    sinks = w["sink"] if c.sink else np.full(H, -np.inf)
    o = ref.causal_attention(q.reshape(n, H, c.dim), k.reshape(n, G, c.dim), v, c.scale, c.softcap or 1.0, sinks,
                             None if c.softcap else "no_cap")
    y = ref.rms_norm(o.reshape(n, -1) @ w["o"].T, (1.0 if cfg.norm_one_plus else 0.0) + np.asarray(t["l0.norm1"], np.float64), cfg.norm_eps)
    return x + y


@pytest.mark.parametrize("on", ["none", "qk_norm", "sink", "softcap", "q_temp", "q_temp_fraction", "plain_norm"])
def test_attention_mechanisms_alone(bt, on):
    c = lay.LayerConfig(A, 4, 24, kv_heads=2, dim=16, qk_norm=int(on == "qk_norm"), sink=int(on == "sink"), scale=0.5,
                        softcap=1.5 if on == "softcap" else 0.0, q_temp_coef=0.7 if on.startswith("q_temp") else 0.0, q_temp_every=8.5 if on == "q_temp_fraction" else 9)
    cfg = lay.LayersConfig(50, 64, 120, 1e-5, on != "plain_norm", [c])
    t = make_tensors(cfg, seed=9)
    tokens = np.random.default_rng(9).integers(0, 50, 70).astype(np.int32)
    want = layer_mix(cfg, t, tokens)
    m = lay.build_layered(cfg, t, dtype="float32")
    m.set_trace(True, rows=70)
    m.prefill(tokens)
    assert row_errors(m.read_trace(70)[0], want).max() <= 1e-5
    m.reset_kv_cache()
    for i, x in enumerate(tokens[:40]):
        m.forward_one([x])
        assert np.abs(m.read_trace(1)[0, 0] - want[i]).max() <= 1e-4
    m.set_trace(False)


def test_recurrence_alone_far_token(bt):
    """A first token far behind still shows: with slow decays the state carries it over hundreds of positions."""
    cfg = lay.LayersConfig(40, 48, 700, 1e-5, True, [ssm(3, 16, 20, taps=4, norm_groups=3)])
    t = make_tensors(cfg, seed=4)
    t["l0.mix.A_log"] = bf16(np.full(3, -6.0))
    rng = np.random.default_rng(4)
    tokens = rng.integers(1, 40, 600).astype(np.int32)
    tokens[0] = 0
    t["embed"] = np.array(t["embed"])
    t["embed"][0] *= 32  # one token of weight
    logits, _ = oracle(cfg, t, tokens)
    other = tokens.copy()
    other[0] = 1
    assert row_errors(oracle(cfg, t, other)[0], logits)[-1] > 100 * TOL["float32"][0]
    for dtype in ("float32", "bfloat16"):
        m = lay.build_layered(cfg, t, dtype=dtype)
        for sizes in ([600], [250, 1, 2, 37], [500] + [1] * 100, [63, 65]):
            m.reset_kv_cache()
            e = row_errors(feed(m, tokens, sizes), logits)
            # where C_t is nearly at right angles to the heavy token's B, bf16 rounding of the two shows at single places
            assert (e.max() <= TOL["float32"][0] if dtype == "float32" else np.sqrt((e * e).mean()) <= 0.02), (sizes, e.max())


def needle_model(n_positions, dtype_seed=0):
    """One attention layer whose query of token 1 points at the key of token 0 (score far above all others)."""
    cfg = lay.LayersConfig(60, 96, n_positions, 1e-5, True, [attn(4, 2, 32, 24, scale=0.6, cap=18.0, coef=0.3, every=50)])
    t = make_tensors(cfg, seed=11 + dtype_seed)
    t["pos"] = bf16(0.05 * np.asarray(t["pos"]))
    e = np.asarray(t["embed"], np.float64)
    wk = np.asarray(t["l0.mix.k"], np.float64).reshape(2, 32, 96)
    wq = np.asarray(t["l0.mix.q"], np.float64).reshape(4, 32, 96)
    for h in range(4):
        wq[h] += 4.0 * np.outer(wk[h // 2] @ e[0], e[1] / (e[1] @ e[1]))
    t["l0.mix.q"] = bf16(wq.reshape(128, 96).astype(np.float32))
    return cfg, t


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_keys_at_tile_borders(bt, dtype):
    cfg, t = needle_model(420)
    rng = np.random.default_rng(2)
    m = lay.build_layered(cfg, t, dtype=dtype)
    for place, asks in ((0, (1, 63, 64, 65, 399)), (63, (64, 127, 128, 300)), (64, (127, 128, 192, 399)), (127, (128, 255, 256)),
                        (128, (129, 383, 384)), (255, (256, 257, 399))):
        tokens = rng.integers(2, 60, 400).astype(np.int32)
        tokens[place] = 0
        for a in asks:
            tokens[a] = 1
        logits, _ = oracle(cfg, t, tokens)
        lost = tokens.copy()
        lost[place] = 2
        away, _ = oracle(cfg, t, lost)
        for a in asks:
            assert row_errors(away, logits)[a] > 0.3, "the needle does not stand out"
        for sizes in ([400], [64], [63, 2], [max(place, 2), 37, 1], [390, 1], [256, 128, 2]):
            m.reset_kv_cache()
            assert_close(feed(m, tokens, sizes), logits, dtype, (place, sizes))
        # decoded alone right behind a prompt that ends at the needle, and at its own position
        m.reset_kv_cache()
        m.prefill_logits(tokens[:place + 1], []) if place else m.prefill(tokens[:1])
        nxt = np.array([1], np.int32)
        got = m.forward_one(nxt)[0]
        want, _ = oracle(cfg, t, np.concatenate([tokens[:place + 1], nxt]))
        assert_close(got, want[-1:], dtype)


@pytest.mark.parametrize("dtype,batch", [("float32", 3), ("bfloat16", 2), ("bfloat16", 8), ("bfloat16", 9), ("float32", 12), ("bfloat16", 21)])
def test_batch_equals_each_alone(bt, dtype, batch):
    cfg, t = CONFIGS["odd"], make_tensors(CONFIGS["odd"], seed=6)
    rng = np.random.default_rng(batch)
    tokens = rng.integers(0, cfg.vocab_size, (batch, 40)).astype(np.int32)
    m = lay.build_layered(cfg, t, max_batch=batch, dtype=dtype)
    got = [m.prefill_logits(tokens[:, :33], np.arange(33))]
    for i in range(33, 40):
        lg, nxt = m.forward_one(tokens[:, i])
        assert np.array_equal(nxt, lg.argmax(1))
        got.append(lg[:, None])
    got = np.concatenate(got, axis=1)
    for b in sorted({0, 1, batch // 2, batch - 1}):
        want, _ = oracle(cfg, t, tokens[b])
        assert_close(got[b], want, dtype, b)


def test_reset_leaves_nothing_behind(bt):
    cfg, t, tokens, _, _ = case("plain")
    fresh = lay.build_layered(cfg, t)
    want = feed(fresh, tokens[:30], [20, 1])
    m = lay.build_layered(cfg, t)
    for first in (tokens[::-1].copy(), tokens[:7]):
        m.reset_kv_cache()
        feed(m, first, [50, 1, 3])
        m.reset_kv_cache()
        assert m.current_pos == 0
        assert np.array_equal(feed(m, tokens[:30], [20, 1]), want)


def test_long_decoding(bt):
    cfg = CONFIGS["odd"]
    t = make_tensors(cfg, seed=8)
    tokens = np.random.default_rng(8).integers(0, cfg.vocab_size, 500).astype(np.int32)
    logits, _ = oracle(cfg, t, tokens)
    for dtype in ("float32", "bfloat16"):
        m = lay.build_layered(cfg, t, dtype=dtype)
        assert_close(feed(m, tokens, [3] + [1] * 497), logits, dtype)
        m.reset_kv_cache()
        assert row_errors(m.prefill_logits(tokens, [0, 250, 499]), logits[[0, 250, 499]]).max() <= TOL[dtype][0]


def test_greedy_generation(bt):
    cfg, t, tokens, _, _ = case("plain")
    m = lay.build_layered(cfg, t, max_batch=2, dtype="float32")
    prompts = np.stack([tokens[:12], tokens[20:32]])
    out = m.generate(prompts, 15)
    for b in range(2):
        seq = list(prompts[b])
        for j in range(15):
            lg = oracle(cfg, t, seq)[0][-1]
            top = np.sort(lg)[-2:]
            assert lg[out[b, j]] >= top[1] - 1e-3 * np.abs(lg).max(), (b, j)  # the pick, or a tie within rounding
            seq.append(int(out[b, j]))
    assert np.array_equal(m.generate(prompts, 15), out)


def test_memory_file_resumes(bt, tmp_path):
    cfg, t, tokens, logits, _ = case("odd")
    a, b = lay.build_layered(cfg, t, dtype="float32"), lay.build_layered(cfg, t, dtype="float32")
    feed(a, tokens[:50], [50])
    a.save_memory(str(tmp_path / "m.safetensors"))
    feed(b, tokens[::-1].copy(), [30])
    b.load_memory(str(tmp_path / "m.safetensors"))
    assert b.current_pos == 50
    got = np.concatenate([b.forward_one(tokens[i:i + 1])[0] for i in range(50, 60)])
    assert_close(got, logits[50:60], "float32")


def test_positions_end_where_the_cache_ends(bt):
    cfg, t, tokens, _, _ = case("wide")
    m = lay.build_layered(cfg, t, max_seq_len=20)
    m.prefill(tokens[:20])
    for call in (lambda: m.forward_one(tokens[20:21]), lambda: m.prefill(tokens[20:22])):
        with pytest.raises(bt.BitTTTError, match="max_position"):
            call()
    with pytest.raises(bt.BitTTTError):
        m.set_layer_tensor(0, 0, np.zeros(cfg.width, np.float32))  # finalized


@pytest.mark.parametrize("rows", [70, 130, 300, 2000])
def test_products_of_many_tiles(bt, rows):
    """Wide layers: several input blocks per warp of the streaming product, several tiles per CTA of the tcgen05 product,
    cut and uncut input ranges, row counts on both sides of every tile size."""
    cfg = lay.LayersConfig(200, 1284, 2048, 1e-5, True, [
        ssm(16, 40, 64, groups=2, norm_groups=4), attn(4, 2, 64, 64, ff=5000)])
    t = make_tensors(cfg, seed=1)
    tokens = np.random.default_rng(rows).integers(0, 200, rows).astype(np.int32)
    want, _ = oracle(cfg, t, tokens, dtype=np.float32)
    m = lay.build_layered(cfg, t)
    ask = np.unique(np.linspace(0, rows - 1, 40).astype(int))
    assert_close(m.prefill_logits(tokens, ask), want[ask], "bfloat16")
    if rows <= 300:
        f = lay.build_layered(cfg, t, dtype="float32")
        assert_close(f.prefill_logits(tokens, ask), want[ask], "float32")
        for x in (m, f):  # decode at this width
            x.reset_kv_cache()
            x.prefill(tokens[:-3])
            got = np.concatenate([x.forward_one(tokens[i:i + 1])[0] for i in range(rows - 3, rows)])
            assert_close(got, want[-3:], "bfloat16" if x is m else "float32")


def test_trace_run_replays_a_checkpoint(bt, tmp_path):
    """bin/trace_run as a user starts it: a process of its own, steps on its standard input."""
    import json
    import os
    import subprocess
    import sys

    from layered_common import ROOT
    cfg, t, tokens, logits, _ = case("odd")
    loader = importlib.import_module("bit-ttt-engine_b200.loader")
    loader.write_safetensors(str(tmp_path / "model.safetensors"), t)
    (tmp_path / "config.json").write_text(json.dumps(lay.gufotar_dict(cfg)))
    (tmp_path / "out").mkdir()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": tokens[:40].tolist(), "want": [0, 39]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": tokens[40:41].tolist(), "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": tokens[41:42].tolist(), "want": [0]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": tokens[:3].tolist(), "want": [2]}], "end": ["b"]}]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32", "--out",
                        str(tmp_path / "out"), "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)), text=True,
                       capture_output=True, timeout=300)
    assert p.returncode == 0, p.stderr
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    assert not (tmp_path / "out" / "1.f32").exists()
    for step, places in ((0, [0, 39]), (2, [41]), (3, [2])):
        got = np.fromfile(tmp_path / "out" / f"{step}.f32", "<f4").reshape(len(places), cfg.vocab_size)
        assert_close(got, logits[places], "float32")
