"""Small configurations and random weights of the design `Fepapel`, and the comparison with oracle/fepapel.py."""
import numpy as np

from layered_common import bf16, lay, row_errors  # noqa: F401  (row_errors: for the tests)
from oracle import fepapel as ref


def moe(ff, experts, top, shared):
    return dict(mlp=lay.MLP_MOE_SWIGLU, ff=ff, experts=experts, top=top, shared_ff=shared)


def latent(heads, dim, rot, vdim, rank, scale=0.25, base=900.0, rot_dims=None, **mlp):
    return lay.LayerConfig(lay.MIX_LATENT, heads, vdim, dim=dim, scale=scale, rot_dim=rot, rot_dims=rot if rot_dims is None else rot_dims,
                           rot_base=base, kv_rank=rank, out_gate=1, **mlp)


def wkv(heads, dim, rank, **mlp):
    return lay.LayerConfig(lay.MIX_WKV, heads, dim=dim, decay_rank=rank, **mlp)


def rglru(channels, blocks, taps, **mlp):
    return lay.LayerConfig(lay.MIX_RGLRU, channels=channels, blocks=blocks, conv_taps=taps, **mlp)


def config(vocab, width, layers, loop=None, eps=1e-5, cap=12.0):
    return lay.LayersConfig(vocab, width, 0, eps, False, layers, pre_norm=True, loop=loop, logit_softcap=cap)


CONFIGS = {
    # a loop in the middle, three passes, a layer without feed-forward inside it
    "loop": config(90, 128, [rglru(96, 3, 4, **moe(32, 6, 2, 48)), latent(4, 32, 16, 24, 40), wkv(2, 32, 8, **moe(40, 5, 3, 16)),
                             latent(2, 16, 8, 16, 64, **moe(24, 4, 1, 32))], loop=(1, 3, 3)),
    # sizes that are no multiples of 8 or 16; the loop takes all layers
    "odd": config(131, 100, [wkv(3, 20, 5, **moe(44, 5, 3, 20)), latent(3, 20, 6, 12, 36, **moe(30, 7, 2, 11)), rglru(60, 4, 6, **moe(17, 3, 2, 29))],
                  loop=(0, 3, 2), eps=3e-6, cap=7.0),
    # no loop; more heads than one tile of heads, several blocks of latents, wide recurrences, one expert per token, no shared expert
    "wide": config(77, 192, [latent(36, 48, 32, 32, 300, scale=0.15, **moe(72, 40, 1, 56)), rglru(320, 1, 1), wkv(1, 128, 70, **moe(64, 9, 9, 0)), wkv(2, 64, 16)]),
    # heads too wide for the tile kernel; part of the rotated dimensions pass; a loop of one pass at the end; many blocks, long and short memory
    "heads": config(64, 96, [latent(2, 224, 40, 72, 130, scale=0.1, rot_dims=24, **moe(16, 3, 3, 64)), rglru(96, 12, 3), wkv(1, 160, 3), latent(18, 8, 2, 8, 16)],
                    loop=(2, 4, 1), eps=1e-4, cap=30.0),
}


def make_tensors(cfg, seed=0, **scale):
    """Random tensors (values representable in bf16).  Decays are spread from fast to slow, so that near and far tokens count."""
    rng = np.random.default_rng(seed)
    t = {}
    for name, shape, layer, _ in lay.tensor_shapes(cfg):
        leaf = name.split(".", 1)[1] if name.startswith("l") and name[1].isdigit() else name
        last, n = leaf.rsplit(".", 1)[-1], rng.normal(0, 1, shape)
        if leaf == "embed":
            a = n
        elif "norm" in last:
            a = 1.0 + 0.2 * n
        elif last == "w0":
            a = rng.uniform(-6.0, 1.0, shape)
        elif last == "lam":
            a = rng.uniform(-7.0, 0.0, shape)
        elif ".mu." in leaf:
            a = rng.uniform(0.0, 1.0, shape)
        elif last in ("b", "u") or leaf == "loop.step":
            a = 0.5 * n
        elif leaf == "mix.conv":
            a = n / np.sqrt(shape[1])
        elif last == "router":
            a = 2.0 * n / np.sqrt(shape[-1])
        else:
            a = n / np.sqrt(shape[-1])
        t[name] = bf16(np.asarray(a, np.float32) * scale.get(leaf, 1.0))
    return t


def oracle(cfg, tensors, tokens, flaw=None, dtype=np.float64):
    return ref.forward(lay.fepapel_dict(cfg), tensors, tokens, dtype=dtype, flaw=flaw)


FLAWS = ("no_shift", "no_bonus", "wkv_state_lost", "short_conv", "rglru_state_lost", "first_key_lost", "own_key_lost", "no_rotation",
         "no_output_gate", "no_shared", "no_router_bias", "no_loop_input", "same_step", "no_post_norm", "no_logit_cap")
