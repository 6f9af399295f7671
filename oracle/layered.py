"""Plain, slow CPU restatement of the layer-list decoder design (`Gufotar`).  TEST INFRASTRUCTURE, NOT PRODUCT CODE.

One function per mechanism, numpy, float64 unless the caller asks for another type, no caching and no
chunking: a whole sequence goes in, every position's values come out.  It shares nothing with the product
path (neither its configuration classes nor its kernels): it reads the same config dictionary and the same
name -> array mapping a checkpoint holds.

A `flaw` argument of :func:`forward` plants one deliberate mistake (a lost sink, a key left out, ...): the tests use
it to show that their inputs would expose such a mistake.
"""
from __future__ import annotations

import numpy as np


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def grouped_rms_norm(x, w, groups, eps):
    """The same over `groups` equal parts of the last axis, each by its own root mean square."""
    t, n = x.shape
    parts = x.reshape(t, groups, n // groups)
    parts = parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return parts.reshape(t, n) * w


def silu(x):
    return x / (1.0 + np.exp(-x))


def softplus(x):
    return np.maximum(x, 0.0) + np.log1p(np.exp(-np.abs(x)))


def relu_squared(x):
    return np.square(np.maximum(x, 0.0))


def query_temperature(positions, coef, every):
    """Factor on the query at each position: grows by coef * ln(steps + 1), one step per `every` positions."""
    steps = np.floor((np.asarray(positions, np.float64) + 1.0) / every)
    return 1.0 + coef * np.log(steps + 1.0)


def capped(score, cap):
    return cap * np.tanh(score / cap)


def sink_softmax(scores, sink):
    """Softmax over the last axis whose denominator has one more term exp(sink)."""
    top = np.maximum(scores.max(axis=-1, keepdims=True), sink)
    e = np.exp(scores - top)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - top))


def causal_attention(q, k, v, scale, cap, sinks, flaw=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv], sinks [H] -> [T, H, dv]; query head h reads key head h // (H / G)."""
    t, heads, _ = q.shape
    rep = heads // k.shape[1]
    out = np.zeros((t, heads, v.shape[2]), q.dtype)
    for h in range(heads):
        g = h // rep
        for i in range(t):
            lo = 1 if flaw == "first_key_lost" and i > 0 else 0
            hi = i if flaw == "own_key_lost" and i > 0 else i + 1
            s = capped((k[lo:hi, g] @ q[i, h]) * scale, cap) if flaw != "no_cap" else (k[lo:hi, g] @ q[i, h]) * scale
            p = sink_softmax(s, -np.inf if flaw == "no_sink" else sinks[h])
            out[i, h] = p @ v[lo:hi, g]
    return out


def attention_mixer(x, w, cfg, eps, v_first, flaw=None):
    """x [T, width] -> (mixed [T, width], v as projected [T, G dv]).  v_first: the first value-mixing layer's
    projected values, or None in that layer and in layers without value mixing."""
    t = x.shape[0]
    H, G, d, dv = cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms_norm(x @ w["q"].T, w["q.norm"], eps)  # over all heads at once
    k = rms_norm(x @ w["k"].T, w["k.norm"], eps)
    v = x @ w["v"].T
    if flaw != "no_temperature":
        q = q * query_temperature(np.arange(t), cfg["q_temp"]["coef"], cfg["q_temp"]["every"]).astype(q.dtype)[:, None]
    mixed = v
    if v_first is not None and flaw != "no_value_mix":
        lam = w["vmix"]
        mixed = (1.0 - lam) * v + lam * v_first
    o = causal_attention(q.reshape(t, H, d), k.reshape(t, G, d), mixed.reshape(t, G, dv), cfg["scale"], cfg["softcap"], w["sink"], flaw)
    return o.reshape(t, H * dv) @ w["o"].T, v


def causal_conv(x, kernel, bias):
    """x [T, C], kernel [C, taps] (last column: the current token), zeros before the start."""
    t, taps = x.shape[0], kernel.shape[1]
    out = np.tile(bias, (t, 1)).astype(x.dtype)
    for j in range(taps):
        back = taps - 1 - j
        out[back:] += x[:max(t - back, 0)] * kernel[:, j]
    return out


def ssm_scan(x, b, c, dt, a_log, d, flaw=None):
    """x [T, heads, P], b and c [T, groups, N], dt [T, heads] -> y [T, heads, P]; token by token.
    S <- exp(-exp(a_log) dt) S + dt b x^T;  y = S^T c + d x."""
    t, heads, p = x.shape
    groups, n = b.shape[1:]
    s = np.zeros((heads, n, p), x.dtype)
    y = np.zeros_like(x)
    for i in range(t):
        if flaw == "state_lost" and i == t // 2:
            s[:] = 0
        for h in range(heads):
            g = h // (heads // groups)
            s[h] = np.exp(-np.exp(a_log[h]) * dt[i, h]) * s[h] + dt[i, h] * np.outer(b[i, g], x[i, h])
            y[i, h] = c[i, g] @ s[h] + d[h] * x[i, h]
    return y


def ssm_mixer(x, w, cfg, eps, flaw=None):
    t = x.shape[0]
    heads, p, n, groups = cfg["heads"], cfg["vdim"], cfg["state"], cfg["groups"]
    inner = heads * p
    proj = x @ w["in"].T
    z, xbc, dt = np.split(proj, [inner, 2 * inner + 2 * groups * n], axis=1)
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    xs, b, c = np.split(xbc, [inner, inner + groups * n], axis=1)
    y = ssm_scan(xs.reshape(t, heads, p), b.reshape(t, groups, n), c.reshape(t, groups, n), softplus(dt + w["dt_bias"]),
                 w["A_log"], w["D"], flaw)
    y = y.reshape(t, inner) * silu(z)
    return grouped_rms_norm(y, w["norm"], cfg["norm_groups"], eps) @ w["o"].T


def sub(weights, prefix, dtype):
    return {k[len(prefix):]: np.asarray(v, dtype) for k, v in weights.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=np.float64, flaw=None):
    """(logits [T, vocab], residual stream after every layer [layers, T, width]) of one sequence."""
    eps = config["norm"]["eps"]
    one = 0.0 if flaw == "plain_norm" else 1.0
    tokens = np.asarray(tokens)
    x = np.asarray(weights["embed"], dtype)[tokens] + np.asarray(weights["pos"], dtype)[:len(tokens)]
    v_first, stream = None, []
    for i, layer in enumerate(config["layers"]):
        w = sub(weights, f"l{i}.mix.", dtype)
        cfg = layer["mixer"]
        if layer["type"] == "attention":
            mixes = bool(cfg["v_mix"])
            m, v = attention_mixer(x, w, cfg, eps, v_first if mixes else None, flaw)
            if mixes and v_first is None:
                v_first = v
        elif layer["type"] == "mamba2":
            m = ssm_mixer(x, w, cfg, eps, flaw)
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(m, one + np.asarray(weights[f"l{i}.norm1"], dtype), eps)
        if layer["mlp"] is not None:
            if layer["mlp"]["kind"] != "dense":
                raise ValueError(layer["mlp"]["kind"])
            up, down = np.asarray(weights[f"l{i}.mlp.up"], dtype), np.asarray(weights[f"l{i}.mlp.down"], dtype)
            f = relu_squared(x @ up.T) @ down.T
            x = x + rms_norm(f, one + np.asarray(weights[f"l{i}.norm2"], dtype), eps)
        stream.append(x)
    logits = rms_norm(x, one + np.asarray(weights["final.norm"], dtype), eps) @ np.asarray(weights["head"], dtype).T
    return logits, np.stack(stream)
