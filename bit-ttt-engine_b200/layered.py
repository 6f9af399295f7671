"""Models given as a list of layers: configuration, checkpoint tensors, registry entry of the `Gufotar` design.

`LayersConfig` / `LayerConfig` describe what the library's layer-list model takes (`bt_layers_config`,
`bt_layer_config`): one mixer per layer - softmax attention with capped scores, a sink, whole-projection query/key norm,
query temperature and value mixing, each switched by its own parameter, or a state-space recurrence - and an optional
dense feed-forward.  A design maps its config.json and its tensor names onto them.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np

from .model import (LT_K, LT_K_NORM, LT_MLP_DOWN, LT_MLP_UP, LT_NORM1, LT_NORM2, LT_O, LT_Q, LT_Q_NORM, LT_SINK,
                    LT_SSM_A_LOG, LT_SSM_CONV, LT_SSM_CONV_B, LT_SSM_D, LT_SSM_DT_BIAS, LT_SSM_IN, LT_SSM_NORM,
                    LT_SSM_O, LT_V, LT_VMIX, LayeredLM, MIX_ATTENTION, MIX_SSM, MLP_DENSE_RELU2, MLP_NONE, T_EMBED,
                    T_LM_HEAD, T_NORM_F, T_POS)


@dataclass
class LayerConfig:
    """One layer; the fields of `bt_layer_config`."""
    mixer: int
    heads: int
    vdim: int
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


@dataclass
class LayersConfig:
    vocab_size: int
    width: int
    max_positions: int
    norm_eps: float
    norm_one_plus: bool = True
    layers: list = field(default_factory=list)


def tensor_shapes(cfg: LayersConfig):
    """[(name, shape, layer or None, slot)] of a checkpoint: layer i's tensors are `l<i>.*`."""
    W, V = cfg.width, cfg.vocab_size
    out = [("embed", (V, W), None, T_EMBED), ("head", (V, W), None, T_LM_HEAD), ("final.norm", (W,), None, T_NORM_F)]
    if cfg.max_positions:
        out.append(("pos", (cfg.max_positions, W), None, T_POS))
    for i, c in enumerate(cfg.layers):
        inner = c.heads * c.vdim
        t = [("norm1", (W,), LT_NORM1)]
        if c.mixer == MIX_ATTENTION:
            nq, nk, nv = c.heads * c.dim, c.kv_heads * c.dim, c.kv_heads * c.vdim
            t += [("mix.q", (nq, W), LT_Q), ("mix.k", (nk, W), LT_K), ("mix.v", (nv, W), LT_V), ("mix.o", (W, inner), LT_O)]
            if c.qk_norm:
                t += [("mix.q.norm", (nq,), LT_Q_NORM), ("mix.k.norm", (nk,), LT_K_NORM)]
            if c.sink:
                t.append(("mix.sink", (c.heads,), LT_SINK))
            if c.v_mix:
                t.append(("mix.vmix", (), LT_VMIX))
        else:
            ch = inner + 2 * c.groups * c.state
            t += [("mix.in", (inner + ch + c.heads, W), LT_SSM_IN), ("mix.conv", (ch, c.conv_taps), LT_SSM_CONV),
                  ("mix.conv.b", (ch,), LT_SSM_CONV_B), ("mix.dt_bias", (c.heads,), LT_SSM_DT_BIAS),
                  ("mix.A_log", (c.heads,), LT_SSM_A_LOG), ("mix.D", (c.heads,), LT_SSM_D),
                  ("mix.norm", (inner,), LT_SSM_NORM), ("mix.o", (W, inner), LT_SSM_O)]
        if c.mlp != MLP_NONE:
            t += [("norm2", (W,), LT_NORM2), ("mlp.up", (c.ff, W), LT_MLP_UP), ("mlp.down", (W, c.ff), LT_MLP_DOWN)]
        out += [(f"l{i}.{name}", shape, i, slot) for name, shape, slot in t]
    return out


# ---------------------------------------------------------------------------------------
# Gufotar
# ---------------------------------------------------------------------------------------

def gufotar_config(d: dict) -> LayersConfig:
    """config.json of a Gufotar checkpoint."""
    from .loader import CheckpointError

    def need(m: dict, key: str, where: str):
        if key not in m:
            raise CheckpointError(f"config: {where}.{key} is missing")
        return m[key]

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
            m.set_layer_tensor(layer, slot, data)
    m.finalize()
    return m


# `architecture` of config.json -> reader of that design's configuration
DESIGNS = {"Gufotar": gufotar_config}
