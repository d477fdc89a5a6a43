"""Small random Derupel models for the tests."""
from __future__ import annotations

import numpy as np

from ytensor_b200.derupel import DECAYED, LATENT, DerupelConfig, DerupelLayer
from ytensor_b200.native_lm import MLP_DENSE, MLP_MOE, MLP_NONE
from ytensor_b200.qwen3 import bf16_bits_to_f32, f32_to_bf16_bits

MLPS = {"dense": MLP_DENSE, "moe": MLP_MOE, None: MLP_NONE}


def decayed(heads=3, dim=24, vdim=40, decay=None, mlp="dense", ff=48, **kw):
    decay = decay or [float(x) for x in np.linspace(0.4, 0.995, heads)]
    return DerupelLayer(mixer=DECAYED, heads=heads, dim=dim, vdim=vdim, decay=decay, mlp=MLPS[mlp], ff=ff if mlp else 0, **kw)


def latent(heads=3, dim=20, rot=12, vdim=28, kv_rank=40, q_rank=52, base=10000.0, scale=None, mlp="dense", ff=48, **kw):
    return DerupelLayer(mixer=LATENT, heads=heads, dim=dim, vdim=vdim, rot_dim=rot, rot_dims=rot, rot_base=base,
                        kv_rank=kv_rank, q_rank=q_rank, scale=(dim + rot) ** -0.5 if scale is None else scale,
                        mlp=MLPS[mlp], ff=ff if mlp else 0, **kw)


def config(layers, width=56, vocab=90, eps=1e-5, scale=2.5):
    return DerupelConfig(width=width, vocab=vocab, eps=eps, embed_scale=scale, layers=layers)


def weights(cfg, seed=0, key_gain=2.0, router_gain=1.5):
    """name -> bf16 bits (what a checkpoint stores). Query and key matrices are scaled up so that single keys stand out of a
    softmax; gates and expert inputs reach their bounds."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        leaf = name.split(".")[-1]
        if leaf.startswith("norm"):
            a = 1 + 0.2 * rng.standard_normal(shape)
        elif leaf == "embed":
            a = rng.standard_normal(shape) / cfg.embed_scale
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if leaf in ("uq", "uk"):
                a = a * key_gain
            if leaf == "router":
                a = a * router_gain
        out[name] = f32_to_bf16_bits(np.asarray(a, np.float32)).reshape(shape)
    return out


def floats(w):
    return {k: bf16_bits_to_f32(v).reshape(np.shape(v)) for k, v in w.items()}


# Configurations with sizes that differ from each other wherever the design lets them: every size that could be mistaken
# for another one shows.
def odd():
    """Sizes that are no multiples of anything, layers of one kind with different sizes and constants, a layer without a
    feed-forward, a mixture without a shared expert, one expert of one, widths that differ between shared and other experts."""
    return config([latent(5, 12, 6, 20, 28, 44, base=700.0, ff=36),
                   decayed(3, 12, 20, mlp="moe", ff=20, experts=5, top=3, limit=0.7, shared_ff=28, shared_limit=1.9),
                   decayed(2, 28, 12, decay=[1.0, 0.05], mlp=None),
                   latent(3, 20, 10, 12, 52, 20, base=30000.0, scale=0.4, mlp="moe", ff=12, experts=1, top=1, limit=2.5),
                   decayed(4, 20, 36, mlp="moe", ff=28, experts=7, top=7, limit=1.1, shared_ff=12, shared_limit=0.4)],
                  width=50, vocab=77, eps=3e-4, scale=3.3)


def mixed():
    """Rotated part larger than the rest, value heads of the tensor-core width, one head; a mixture behind each mixer."""
    return config([decayed(2, 64, 64, ff=72),
                   latent(4, 16, 48, 64, 96, 72, mlp="moe", ff=40, experts=9, top=2, limit=1.0, shared_ff=24,
                          shared_limit=1.0),
                   decayed(1, 128, 128, mlp="moe", ff=24, experts=6, top=1, limit=1.3, shared_ff=40, shared_limit=0.8),
                   latent(1, 32, 32, 32, 64, 32, scale=0.3, ff=64)], width=64, vocab=130)


def wide():
    """Heads of the tensor-core attention's larger tile, more heads than share one pass over the cache, a latent wider than
    a warp's load."""
    return config([latent(18, 40, 40, 72, 272, 136, ff=200),
                   decayed(6, 96, 128, ff=104),
                   latent(2, 64, 64, 128, 528, 64, base=500.0, mlp="moe", ff=72, experts=6, top=2, limit=1.5, shared_ff=72,
                          shared_limit=1.5),
                   decayed(2, 160, 136, ff=40)], width=264, vocab=301)


CONFIGS = {"odd": odd, "mixed": mixed, "wide": wide}
