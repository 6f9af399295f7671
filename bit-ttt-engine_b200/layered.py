"""Models given as a list of layers: configuration, checkpoint tensors, registry entries of the designs `Gufotar` and
`Fepapel`.

`LayersConfig` / `LayerConfig` describe what the library's layer-list model takes (`bt_layers_config`,
`bt_layer_config`): one mixer per layer - softmax attention with capped scores, a sink, whole-projection query/key norm,
query temperature and value mixing, each switched by its own parameter; latent attention with a rotated key part and an
output gate; a state-space, a wkv or a gated linear recurrence - and an optional feed-forward, dense or a mixture of
experts; norms behind and, by design, in front of every sublayer; a looped run of layers.  A design maps its config.json
and its tensor names onto them.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np

from . import model as M
from .model import LayeredLM, MIX_ATTENTION, MIX_LATENT, MIX_RGLRU, MIX_SSM, MIX_WKV, MLP_DENSE_RELU2, MLP_MOE_SWIGLU, MLP_NONE


@dataclass
class LayerConfig:
    """One layer; the fields of `bt_layer_config`."""
    mixer: int
    heads: int = 0
    vdim: int = 0
    # attention
    kv_heads: int = 0
    dim: int = 0
    qk_norm: int = 0
    sink: int = 0
    v_mix: int = 0
    scale: float = 1.0
    softcap: float = 0.0
    q_temp_coef: float = 0.0
    q_temp_every: float = 1.0
    # recurrence
    state: int = 0
    groups: int = 0
    conv_taps: int = 0
    norm_groups: int = 0
    # feed-forward
    mlp: int = MLP_NONE
    ff: int = 0
    experts: int = 0
    top: int = 0
    shared_ff: int = 0
    # latent attention
    rot_dim: int = 0
    rot_dims: int = 0
    kv_rank: int = 0
    out_gate: int = 0
    rot_base: float = 10000.0
    # wkv recurrence
    decay_rank: int = 0
    # gated linear recurrence
    channels: int = 0
    blocks: int = 0


@dataclass
class LayersConfig:
    vocab_size: int
    width: int
    max_positions: int
    norm_eps: float
    norm_one_plus: bool = True
    layers: list = field(default_factory=list)
    pre_norm: bool = False
    loop: tuple | None = None  # (first layer, layer behind the last, passes)
    logit_softcap: float = 0.0

    def runs(self) -> list:
        """The layer of every layer run, in the order they run."""
        n = len(self.layers)
        if not self.loop:
            return list(range(n))
        start, stop, times = self.loop
        return list(range(start)) + list(range(start, stop)) * times + list(range(stop, n))


def mixer_tensors(cfg: LayersConfig, c: LayerConfig):
    """[(name, shape, slot)] of a layer's mixer."""
    W = cfg.width
    if c.mixer == MIX_ATTENTION:
        nq, nk, nv, inner = c.heads * c.dim, c.kv_heads * c.dim, c.kv_heads * c.vdim, c.heads * c.vdim
        t = [("q", (nq, W), M.LT_Q), ("k", (nk, W), M.LT_K), ("v", (nv, W), M.LT_V), ("o", (W, inner), M.LT_O)]
        if c.qk_norm:
            t += [("q.norm", (nq,), M.LT_Q_NORM), ("k.norm", (nk,), M.LT_K_NORM)]
        if c.sink:
            t.append(("sink", (c.heads,), M.LT_SINK))
        if c.v_mix:
            t.append(("vmix", (), M.LT_VMIX))
        return t
    if c.mixer == MIX_SSM:
        inner = c.heads * c.vdim
        ch = inner + 2 * c.groups * c.state
        return [("in", (inner + ch + c.heads, W), M.LT_SSM_IN), ("conv", (ch, c.conv_taps), M.LT_SSM_CONV),
                ("conv.b", (ch,), M.LT_SSM_CONV_B), ("dt_bias", (c.heads,), M.LT_SSM_DT_BIAS),
                ("A_log", (c.heads,), M.LT_SSM_A_LOG), ("D", (c.heads,), M.LT_SSM_D),
                ("norm", (inner,), M.LT_SSM_NORM), ("o", (W, inner), M.LT_SSM_O)]
    if c.mixer == MIX_LATENT:
        H = c.heads
        t = [("q", (H * (c.dim + c.rot_dim), W), M.LT_Q), ("dkv", (c.kv_rank + c.rot_dim, W), M.LT_DKV),
             ("dkv.norm", (c.kv_rank,), M.LT_DKV_NORM), ("uk", (H * c.dim, c.kv_rank), M.LT_UK),
             ("uv", (H * c.vdim, c.kv_rank), M.LT_UV), ("o", (W, H * c.vdim), M.LT_O)]
        return t + ([("g", (H, W), M.LT_GATE)] if c.out_gate else [])
    if c.mixer == MIX_WKV:
        n = c.heads * c.dim
        t = [(f"mu.{x}", (W,), slot) for x, slot in zip("rkvgw", (M.LT_MU_R, M.LT_MU_K, M.LT_MU_V, M.LT_MU_G, M.LT_MU_W))]
        t += [(x, (n, W), slot) for x, slot in zip("rkvg", (M.LT_WKV_R, M.LT_WKV_K, M.LT_WKV_V, M.LT_WKV_G))]
        return t + [("w1", (c.decay_rank, W), M.LT_WKV_W1), ("w2", (n, c.decay_rank), M.LT_WKV_W2), ("w0", (n,), M.LT_WKV_W0),
                    ("u", (c.heads, c.dim), M.LT_WKV_U), ("norm", (n,), M.LT_WKV_NORM), ("o", (W, n), M.LT_O)]
    ch, part = c.channels, c.channels // c.blocks
    square, bias = (c.blocks, part, part), (c.blocks, part)
    return [("y", (ch, W), M.LT_RG_Y), ("y.b", (ch,), M.LT_RG_Y_B), ("x", (ch, W), M.LT_RG_X), ("x.b", (ch,), M.LT_RG_X_B),
            ("conv", (ch, c.conv_taps), M.LT_RG_CONV), ("conv.b", (ch,), M.LT_RG_CONV_B), ("ra", square, M.LT_RG_RA),
            ("ra.b", bias, M.LT_RG_RA_B), ("ri", square, M.LT_RG_RI), ("ri.b", bias, M.LT_RG_RI_B), ("lam", (ch,), M.LT_RG_LAM),
            ("o", (W, ch), M.LT_O)]


def mlp_tensors(cfg: LayersConfig, c: LayerConfig):
    """[(name, shape, slot)] of a layer's feed-forward; slot (kind, expert) for an expert's matrix."""
    W = cfg.width
    if c.mlp == MLP_DENSE_RELU2:
        return [("up", (c.ff, W), M.LT_MLP_UP), ("down", (W, c.ff), M.LT_MLP_DOWN)]
    if c.mlp != MLP_MOE_SWIGLU:
        return []
    t = [("router", (c.experts, W), M.LT_ROUTER), ("router.b", (c.experts,), M.LT_ROUTER_B)]
    for e in range(c.experts):
        t += [(f"e{e}.gate", (c.ff, W), (M.LT_E_GATE, e)), (f"e{e}.up", (c.ff, W), (M.LT_E_UP, e)), (f"e{e}.down", (W, c.ff), (M.LT_E_DOWN, e))]
    if c.shared_ff:
        t += [("shared.gate", (c.shared_ff, W), M.LT_S_GATE), ("shared.up", (c.shared_ff, W), M.LT_S_UP), ("shared.down", (W, c.shared_ff), M.LT_S_DOWN)]
    return t


def tensor_shapes(cfg: LayersConfig):
    """[(name, shape, layer or None, slot)] of a checkpoint: layer i's tensors are `l<i>.*`.  norm1 / norm2 stand behind the
    sublayers, or in front of them where there are norms on both sides (then norm1b / norm2b stand behind)."""
    W, V = cfg.width, cfg.vocab_size
    out = [("embed", (V, W), None, M.T_EMBED), ("head", (V, W), None, M.T_LM_HEAD), ("final.norm", (W,), None, M.T_NORM_F)]
    if cfg.max_positions:
        out.append(("pos", (cfg.max_positions, W), None, M.T_POS))
    if cfg.loop:
        out += [("loop.in", (W, 2 * W), None, M.T_LOOP_IN), ("loop.step", (cfg.loop[2], W), None, M.T_LOOP_STEP)]
    for i, c in enumerate(cfg.layers):
        norms = [("norm1", M.LT_NORM1), ("norm2", M.LT_NORM2)]
        if cfg.pre_norm:
            norms = [("norm1", M.LT_PRE1), ("norm2", M.LT_PRE2), ("norm1b", M.LT_NORM1), ("norm2b", M.LT_NORM2)]
        t = [(name, (W,), slot) for name, slot in norms if c.mlp != MLP_NONE or name.startswith("norm1")]
        t += [(f"mix.{name}", shape, slot) for name, shape, slot in mixer_tensors(cfg, c)]
        t += [(f"mlp.{name}", shape, slot) for name, shape, slot in mlp_tensors(cfg, c)]
        out += [(f"l{i}.{name}", shape, i, slot) for name, shape, slot in t]
    return out


def need(m: dict, key: str, where: str):
    """An entry a configuration has to have."""
    from .loader import CheckpointError
    if not isinstance(m, dict) or key not in m:
        raise CheckpointError(f"config: {where}.{key} is missing")
    return m[key]


# ---------------------------------------------------------------------------------------
# Gufotar
# ---------------------------------------------------------------------------------------

def gufotar_config(d: dict, tensors: dict | None = None) -> LayersConfig:
    """config.json of a Gufotar checkpoint."""
    from .loader import CheckpointError

    cfg = LayersConfig(vocab_size=int(need(d, "vocab", "")), width=int(need(d, "width", "")),
                       max_positions=int(need(d, "max_positions", "")), norm_eps=float(need(need(d, "norm", ""), "eps", "norm")))
    for i, entry in enumerate(need(d, "layers", "")):
        where = f"layers[{i}]"
        m, kind = need(entry, "mixer", where), need(entry, "type", where)
        if kind == "attention":
            temp = m.get("q_temp") or {"coef": 0.0, "every": 1.0}
            layer = LayerConfig(MIX_ATTENTION, int(need(m, "heads", where)), int(need(m, "vdim", where)),
                                kv_heads=int(need(m, "kv_heads", where)), dim=int(need(m, "dim", where)), qk_norm=1, sink=1,
                                v_mix=int(bool(m.get("v_mix", False))), scale=float(need(m, "scale", where)),
                                softcap=float(m.get("softcap") or 0.0), q_temp_coef=float(need(temp, "coef", where)),
                                q_temp_every=float(need(temp, "every", where)))
        elif kind == "mamba2":
            layer = LayerConfig(MIX_SSM, int(need(m, "heads", where)), int(need(m, "vdim", where)),
                                state=int(need(m, "state", where)), groups=int(need(m, "groups", where)),
                                conv_taps=int(need(m, "conv", where)), norm_groups=int(need(m, "norm_groups", where)))
        else:
            raise CheckpointError(f"config: {where} has mixer type {kind!r} (attention and mamba2 are known)")
        mlp = entry.get("mlp")
        if mlp is not None:
            if need(mlp, "kind", where) != "dense":
                raise CheckpointError(f"config: {where} has feed-forward kind {mlp['kind']!r} (dense is known)")
            layer.mlp, layer.ff = MLP_DENSE_RELU2, int(need(mlp, "ff", where))
        cfg.layers.append(layer)
    return cfg


def gufotar_dict(cfg: LayersConfig) -> dict:
    """The config.json that `gufotar_config` reads back."""
    layers = []
    for c in cfg.layers:
        if c.mixer == MIX_ATTENTION:
            m = {"heads": c.heads, "kv_heads": c.kv_heads, "dim": c.dim, "vdim": c.vdim, "scale": c.scale, "softcap": c.softcap,
                 "q_temp": {"coef": c.q_temp_coef, "every": c.q_temp_every}, "v_mix": bool(c.v_mix)}
        else:
            m = {"heads": c.heads, "vdim": c.vdim, "state": c.state, "groups": c.groups, "conv": c.conv_taps,
                 "norm_groups": c.norm_groups}
        layers.append({"type": "attention" if c.mixer == MIX_ATTENTION else "mamba2", "mixer": m,
                       "mlp": {"kind": "dense", "ff": c.ff} if c.mlp != MLP_NONE else None})
    return {"architecture": "Gufotar", "vocab": cfg.vocab_size, "width": cfg.width, "max_positions": cfg.max_positions,
            "norm": {"eps": cfg.norm_eps}, "layers": layers}


# ---------------------------------------------------------------------------------------
# Fepapel
# ---------------------------------------------------------------------------------------

def fepapel_config(d: dict, tensors: dict | None = None) -> LayersConfig:
    """config.json of a Fepapel checkpoint.  The decays' rank of a wkv mixer is a size that only its tensors tell."""
    from .loader import CheckpointError
    cfg = LayersConfig(vocab_size=int(need(d, "vocab", "")), width=int(need(d, "width", "")), max_positions=0,
                       norm_eps=float(need(need(d, "norm", ""), "eps", "norm")), norm_one_plus=False, pre_norm=True,
                       logit_softcap=float(d.get("logit_softcap") or 0.0))
    loop = d.get("loop")
    if loop:
        cfg.loop = tuple(int(need(loop, key, "loop")) for key in ("start", "stop", "times"))
    for i, entry in enumerate(need(d, "layers", "")):
        where = f"layers[{i}]"
        m, kind = need(entry, "mixer", where), need(entry, "type", where)

        def size(key, at=m):
            return int(need(at, key, where))

        if kind == "wkv":
            w1 = (tensors or {}).get(f"l{i}.mix.w1")
            if w1 is None:
                raise CheckpointError(f"checkpoint: tensor l{i}.mix.w1 is missing")
            layer = LayerConfig(MIX_WKV, size("heads"), dim=size("dim"), decay_rank=int(np.shape(w1)[0]))
        elif kind == "rglru":
            layer = LayerConfig(MIX_RGLRU, channels=size("width"), blocks=size("blocks"), conv_taps=size("conv"))
        elif kind == "latent_attention":
            rot = need(m, "rot", where)
            layer = LayerConfig(MIX_LATENT, size("heads"), size("vdim"), dim=size("dim"), scale=float(need(m, "scale", where)), rot_dim=size("rot_dim"),
                                rot_dims=size("dims", rot), rot_base=float(need(rot, "base", where)), kv_rank=size("kv_rank"), out_gate=1)
        else:
            raise CheckpointError(f"config: {where} has mixer type {kind!r} (wkv, rglru and latent_attention are known)")
        mlp = entry.get("mlp")
        if mlp is not None:
            if need(mlp, "kind", where) != "moe":
                raise CheckpointError(f"config: {where} has feed-forward kind {mlp['kind']!r} (moe is known)")
            router, shared = need(mlp, "router", where), mlp.get("shared")
            layer.mlp, layer.ff = MLP_MOE_SWIGLU, size("ff", need(mlp, "expert", where))
            layer.experts, layer.top = size("experts", router), size("top", router)
            layer.shared_ff = size("ff", shared) if shared else 0
        cfg.layers.append(layer)
    return cfg


def fepapel_dict(cfg: LayersConfig) -> dict:
    """The config.json that `fepapel_config` reads back."""
    layers = []
    for c in cfg.layers:
        if c.mixer == MIX_WKV:
            kind, m = "wkv", {"heads": c.heads, "dim": c.dim}
        elif c.mixer == MIX_RGLRU:
            kind, m = "rglru", {"width": c.channels, "blocks": c.blocks, "conv": c.conv_taps}
        else:
            kind, m = "latent_attention", {"heads": c.heads, "dim": c.dim, "rot_dim": c.rot_dim, "vdim": c.vdim, "kv_rank": c.kv_rank,
                                           "scale": c.scale, "rot": {"base": c.rot_base, "dims": c.rot_dims}}
        mlp = None
        if c.mlp != MLP_NONE:
            mlp = {"kind": "moe", "expert": {"ff": c.ff}, "router": {"experts": c.experts, "top": c.top},
                   "shared": {"ff": c.shared_ff} if c.shared_ff else None}
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    loop = dict(zip(("start", "stop", "times"), cfg.loop)) if cfg.loop else None
    return {"architecture": "Fepapel", "vocab": cfg.vocab_size, "width": cfg.width, "norm": {"eps": cfg.norm_eps},
            "logit_softcap": cfg.logit_softcap, "loop": loop, "layers": layers}


# ---------------------------------------------------------------------------------------
# checkpoint -> device model
# ---------------------------------------------------------------------------------------

def build_layered(cfg: LayersConfig, tensors: dict, max_batch: int = 1, device: int = 0, dtype: str = "bfloat16",
                  max_seq_len: int | None = None) -> LayeredLM:
    """The device model from a name -> array mapping (a checkpoint's tensors)."""
    from .loader import CheckpointError
    shapes = tensor_shapes(cfg)
    for name, shape, _, _ in shapes:
        if name not in tensors:
            raise CheckpointError(f"checkpoint: tensor {name} is missing")
        if tuple(np.shape(tensors[name])) != shape:
            raise CheckpointError(f"checkpoint: {name} has shape {tuple(np.shape(tensors[name]))}, expected {shape}")
    m = LayeredLM(cfg, max_batch=max_batch, device=device, dtype=dtype, max_seq_len=max_seq_len)
    for name, _, layer, slot in shapes:
        data = np.asarray(tensors[name], np.float32)
        if layer is None:
            m.set_tensor(slot, data)
        else:
            kind, expert = slot if isinstance(slot, tuple) else (slot, None)
            m.set_layer_tensor(layer, kind, data, expert)
    m.finalize()
    return m


# `architecture` of config.json -> reader of that design's configuration
DESIGNS = {"Gufotar": gufotar_config, "Fepapel": fepapel_config}
