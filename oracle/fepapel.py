"""Plain, slow CPU restatement of the layer-list design `Fepapel`.  TEST INFRASTRUCTURE, NOT PRODUCT CODE.

One function per mechanism, numpy, float64 unless the caller asks for another type, no caching and no chunking: a whole
sequence goes in, every position's values come out.  It shares nothing with the product path: it reads the config
dictionary and the name -> array mapping a checkpoint holds.

`flaw` plants one deliberate mistake, so that a test can show that its inputs would expose it.
"""
from __future__ import annotations

import numpy as np

from .layered import causal_conv, rms_norm, silu, softplus, sub


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def gelu_tanh(x):
    return 0.5 * x * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (x + 0.044715 * x ** 3)))


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rotate_pairs(x, positions, base, dims):
    """x [T, ..., d]: neighbouring dimensions (2i, 2i + 1), i < dims / 2, turned by position * base^(-2i/dims)."""
    out = np.array(x)
    i = np.arange(dims // 2)
    angle = np.asarray(positions, np.float64)[:, None] * float(base) ** (-2.0 * i / dims)
    angle = angle.reshape(angle.shape[:1] + (1,) * (x.ndim - 2) + angle.shape[1:])
    c, s = np.cos(angle).astype(x.dtype), np.sin(angle).astype(x.dtype)
    a, b = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = a * c - b * s
    out[..., 1:dims:2] = b * c + a * s
    return out


def shifted(h):
    """Every row's predecessor, zeros in front of the first."""
    return np.concatenate([np.zeros_like(h[:1]), h[:-1]])


def wkv_scan(r, k, v, w, u, flaw=None):
    """r, k, w [T, H, D] (w: decays), v [T, H, D], u [H, D] -> o [T, H, D], token by token."""
    t, heads, d = r.shape
    s = np.zeros((heads, d, v.shape[2]), r.dtype)
    o = np.zeros_like(v)
    for i in range(t):
        if flaw == "wkv_state_lost" and i == t // 2:
            s[:] = 0
        kv = k[i][:, :, None] * v[i][:, None, :]
        bonus = kv if flaw == "no_bonus" else u[:, :, None] * kv
        o[i] = np.einsum("hd,hde->he", r[i], s + bonus)
        s = w[i][:, :, None] * s + kv
    return o


def wkv_mixer(h, w, cfg, eps, flaw=None):
    t, heads, d = h.shape[0], cfg["heads"], cfg["dim"]
    prev = np.zeros_like(h) if flaw == "no_shift" else shifted(h)
    mix = {s: h + (prev - h) * w["mu." + s] for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[s].T).reshape(t, heads, d) for s in "rkv")
    gate = silu(mix["g"] @ w["g"].T)
    decay = np.exp(-np.exp(np.tanh(mix["w"] @ w["w1"].T) @ w["w2"].T + w["w0"])).reshape(t, heads, d)
    o = wkv_scan(r, k, v, decay, w["u"], flaw)
    return (unit_rms(o, eps).reshape(t, heads * d) * w["norm"] * gate) @ w["o"].T


def block_product(x, w, b):
    """x [T, B n], w [B, n, n] ([out, in]), b [B, n]: every part by its own square matrix."""
    t, (blocks, n, _) = x.shape[0], w.shape
    return (np.einsum("tbi,boi->tbo", x.reshape(t, blocks, n), w) + b).reshape(t, blocks * n)


def rglru_scan(u, r, i, lam, flaw=None):
    """S <- a S + sqrt(1 - a^2) i u with a = exp(-8 r softplus(lam)); all states [T, C]."""
    a = np.exp(-8.0 * r * softplus(lam))
    x = np.sqrt(-np.expm1(2.0 * (-8.0 * r * softplus(lam)))) * i * u
    s, out = np.zeros_like(u[0]), np.zeros_like(u)
    for t in range(u.shape[0]):
        if flaw == "rglru_state_lost" and t == u.shape[0] // 2:
            s = np.zeros_like(s)
        s = a[t] * s + x[t]
        out[t] = s
    return out


def rglru_mixer(h, w, cfg, flaw=None):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = causal_conv(h @ w["x"].T + w["x.b"], w["conv"] if flaw != "short_conv" else w["conv"] * (np.arange(w["conv"].shape[1]) > 0), w["conv.b"])
    r = sigmoid(block_product(u, w["ra"], w["ra.b"]))
    i = sigmoid(block_product(u, w["ri"], w["ri.b"]))
    return (rglru_scan(u, r, i, w["lam"], flaw) * y) @ w["o"].T


def causal_softmax_attention(q, k, v, scale, flaw=None):
    """q, k [T, H, d], v [T, H, dv] -> [T, H, dv]."""
    t = q.shape[0]
    seen = np.tril(np.ones((t, t), bool))
    if flaw == "first_key_lost":
        seen[1:, 0] = False
    if flaw == "own_key_lost":
        seen[np.arange(1, t), np.arange(1, t)] = False
    s = np.where(seen[None], np.einsum("ihd,jhd->hij", q, k) * scale, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return np.einsum("hij,jhe->ihe", p / p.sum(-1, keepdims=True), v)


def latent_attention_mixer(h, w, cfg, eps, flaw=None):
    t, H, d, rd, dv, rank = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    pos, rot = np.arange(t), cfg["rot"]
    q = (h @ w["q"].T).reshape(t, H, d + rd)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    qr, kr = q[..., d:], down[:, rank:]
    if flaw != "no_rotation":
        qr, kr = rotate_pairs(qr, pos, rot["base"], rot["dims"]), rotate_pairs(kr, pos, rot["base"], rot["dims"])
    k = np.concatenate([(c @ w["uk"].T).reshape(t, H, d), np.broadcast_to(kr[:, None], (t, H, rd))], axis=-1)
    o = causal_softmax_attention(np.concatenate([q[..., :d], qr], axis=-1), k, (c @ w["uv"].T).reshape(t, H, dv), cfg["scale"], flaw)
    if flaw != "no_output_gate":
        o = o * sigmoid(h @ w["g"].T)[..., None]
    return o.reshape(t, H * dv) @ w["o"].T


def gated_mlp(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def moe(h, w, cfg, flaw=None):
    top = cfg["router"]["top"]
    z = h @ w["router"].T + (0.0 if flaw == "no_router_bias" else w["router.b"])
    out = gated_mlp(h, w, "shared.") if cfg.get("shared") and flaw != "no_shared" else np.zeros((h.shape[0], h.shape[1]), h.dtype)
    for i in range(h.shape[0]):
        best = np.argsort(-z[i], kind="stable")[:top]
        p = np.exp(z[i, best] - z[i, best].max())
        for e, weight in zip(best, p / p.sum()):
            out[i] = out[i] + weight * gated_mlp(h[i:i + 1], w, f"e{e}.")[0]
    return out


def layer_runs(config):
    """[(layer, pass or None)] in the order they run; the pass is given where a pass begins."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


def forward(config, weights, tokens, dtype=np.float64, flaw=None):
    """(logits [T, vocab], residual stream after every layer run [runs, T, width]) of one sequence."""
    eps = config["norm"]["eps"]
    T = {k: np.asarray(v, dtype) for k, v in weights.items()}
    x0 = x = T["embed"][np.asarray(tokens)]
    stream = []
    for i, t in layer_runs(config):
        layer, p = config["layers"][i], f"l{i}."
        if t is not None:
            x = np.concatenate([x, np.zeros_like(x0) if flaw == "no_loop_input" else x0], axis=1) @ T["loop.in"].T
            x = x + T["loop.step"][0 if flaw == "same_step" else t]
        w = sub(T, p + "mix.", dtype)
        h = rms_norm(x, T[p + "norm1"], eps)
        if layer["type"] == "wkv":
            m = wkv_mixer(h, w, layer["mixer"], eps, flaw)
        elif layer["type"] == "rglru":
            m = rglru_mixer(h, w, layer["mixer"], flaw)
        elif layer["type"] == "latent_attention":
            m = latent_attention_mixer(h, w, layer["mixer"], eps, flaw)
        else:
            raise ValueError(layer["type"])
        x = x + (m if flaw == "no_post_norm" else rms_norm(m, T[p + "norm1b"], eps))
        if layer["mlp"] is not None:
            if layer["mlp"]["kind"] != "moe":
                raise ValueError(layer["mlp"]["kind"])
            f = moe(rms_norm(x, T[p + "norm2"], eps), sub(T, p + "mlp.", dtype), layer["mlp"], flaw)
            x = x + rms_norm(f, T[p + "norm2b"], eps)
        stream.append(x)
    logits = rms_norm(x, T["final.norm"], eps) @ T["head"].T
    cap = config["logit_softcap"]
    return (logits if flaw == "no_logit_cap" else cap * np.tanh(logits / cap)), np.stack(stream)
