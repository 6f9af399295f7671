"""Small layer-list configurations and random weights for the tests of that model family, and the comparisons with the
plain implementation in oracle/layered.py."""
import importlib
import os
import sys

import numpy as np

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
if ROOT not in sys.path:
    sys.path.insert(0, ROOT)
from oracle import layered as ref  # noqa: E402

lay = importlib.import_module("bit-ttt-engine_b200.layered")
A, S, RELU2 = lay.MIX_ATTENTION, lay.MIX_SSM, lay.MLP_DENSE_RELU2


def attn(heads, kv, dim, vdim, ff=0, v_mix=1, scale=0.2, cap=15.0, coef=0.25, every=11):
    return lay.LayerConfig(A, heads, vdim, kv_heads=kv, dim=dim, qk_norm=1, sink=1, v_mix=v_mix, scale=scale, softcap=cap,
                           q_temp_coef=coef, q_temp_every=every, mlp=RELU2 if ff else 0, ff=ff)


def ssm(heads, vdim, state, groups=1, taps=4, norm_groups=1, ff=0):
    return lay.LayerConfig(S, heads, vdim, state=state, groups=groups, conv_taps=taps, norm_groups=norm_groups,
                           mlp=RELU2 if ff else 0, ff=ff)


CONFIGS = {
    # grouped heads, sizes that are no multiples of 8 or 16, several groups, feed-forward behind the recurrence
    "odd": lay.LayersConfig(131, 100, 700, 3e-6, True, [
        ssm(4, 20, 24, groups=2, taps=4, norm_groups=4, ff=72), attn(6, 2, 24, 40, ff=136), ssm(6, 9, 7, groups=3, taps=2, norm_groups=3),
        attn(6, 2, 20, 40, v_mix=1, scale=0.3, cap=8.0, coef=0.6, every=7)]),
    # one query head per key head; value mixing starts at the second attention layer; no conv history (one tap)
    "plain": lay.LayersConfig(96, 128, 400, 1e-5, True, [
        attn(2, 2, 64, 64, v_mix=0), attn(3, 3, 64, 32, ff=192), ssm(3, 64, 128, taps=1, norm_groups=3), attn(2, 1, 128, 96, scale=0.1, cap=40.0),
        ssm(2, 100, 64, taps=3, ff=64)]),
    # many query heads per key head, wide heads, odd value size, long convolution
    "wide": lay.LayersConfig(77, 72, 300, 1e-4, True, [
        attn(12, 1, 200, 7, coef=0.1, every=100), ssm(2, 33, 200, groups=1, taps=6), attn(5, 1, 144, 7, ff=80, coef=0.0)]),
    # wide values
    "values": lay.LayersConfig(64, 96, 300, 1e-5, True, [attn(4, 2, 32, 200, ff=96), attn(10, 5, 256, 80, cap=3.0), ssm(5, 16, 16, groups=5, taps=4, norm_groups=5)]),
}


def make_tensors(cfg, seed=0, **scale):
    """Random tensors (values representable in bf16).  The recurrences forget slowly enough for far tokens to matter."""
    rng = np.random.default_rng(seed)
    t = {}
    for name, shape, layer, _ in lay.tensor_shapes(cfg):
        leaf = name.split(".", 1)[1] if name.startswith("l") and "." in name else name
        n = rng.normal(0, 1, shape)
        if leaf in ("embed", "pos"):
            a = n * (1.0 if leaf == "embed" else 0.5)
        elif leaf in ("norm1", "norm2", "final.norm", "norm") :
            a = 0.2 * n
        elif leaf in ("mix.q.norm", "mix.k.norm", "mix.norm", "mix.D"):
            a = 1.0 + 0.2 * n
        elif leaf == "mix.sink":
            a = 1.0 + n
        elif leaf == "mix.vmix":
            a = np.asarray(0.35)
        elif leaf == "mix.A_log":
            a = rng.uniform(-3.0, 0.5, shape)
        elif leaf == "mix.dt_bias":
            a = rng.uniform(-3.0, 0.0, shape)
        elif leaf == "mix.conv":
            a = n / np.sqrt(shape[1])
        elif leaf == "mix.conv.b":
            a = 0.3 * n
        else:
            a = n / np.sqrt(shape[-1])
        t[name] = bf16(np.asarray(a, np.float32) * scale.get(leaf, 1.0))
    return t


def bf16(a):
    u = np.ascontiguousarray(a, np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000).astype(np.uint32).view(np.float32).reshape(np.shape(a))


def oracle(cfg, tensors, tokens, flaw=None, dtype=np.float64):
    return ref.forward(lay.gufotar_dict(cfg), tensors, tokens, dtype=dtype, flaw=flaw)


def row_errors(got, want):
    """Per position: root mean square of the difference (mean taken off) over that of the expected values."""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    w = want - want.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(-1)) / np.sqrt((w * w).mean())
