"""Small random Duzozen models for the tests."""
from __future__ import annotations

import numpy as np

from ytensor_b200.duzozen import MLP_DENSE, MLP_MOE, MLP_NONE, DuzozenConfig, DuzozenLayer
from ytensor_b200.qwen3 import bf16_bits_to_f32, f32_to_bf16_bits


def layer(heads=4, kv=2, dim=16, vdim=16, window=0, cap=12.0, scale=None, v_mix=True, mlp="dense", ff=40, experts=0,
          identity=0, top=0, groups=1, keep=1):
    return DuzozenLayer(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=dim ** -0.5 if scale is None else scale,
                        softcap=cap, window=window, v_mix=v_mix,
                        mlp={"dense": MLP_DENSE, "moe": MLP_MOE, None: MLP_NONE}[mlp], ff=ff if mlp else 0,
                        experts=experts, identity=identity, top=top, groups=groups, keep=keep)


def config(layers, width=48, vocab=90, eps=1e-5):
    return DuzozenConfig(width=width, vocab=vocab, eps=eps, layers=layers)


def weights(cfg, seed=0, qk_gain=2.5, router_gain=2.0):
    """name -> bf16 bits (what a checkpoint stores). Queries and keys are scaled up so that single keys stand out of a
    softmax; the choice correction is as large as the scores, of both signs, so that it decides choices."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        leaf = name.split(".")[-1]
        if leaf == "vmix":
            a = np.float32(rng.uniform(0.2, 0.8))
        elif leaf.startswith("norm") or name == "final.norm":
            a = 1 + 0.2 * rng.standard_normal(shape)
        elif leaf == "correction":
            a = 0.2 * rng.standard_normal(shape) - 0.15
        elif leaf == "embed":
            a = rng.standard_normal(shape)
        else:
            a = rng.standard_normal(shape) / np.sqrt(shape[-1])
            if name.endswith(("mix.q", "mix.k")):
                a = a * qk_gain
            if leaf == "router":
                a = a * router_gain
        out[name] = f32_to_bf16_bits(np.asarray(a, np.float32)).reshape(shape)
    return out


def floats(w):
    return {k: bf16_bits_to_f32(v).reshape(np.shape(v)) for k, v in w.items()}


# Configurations with sizes that differ from each other wherever the design lets them: every size that could be mistaken
# for another one shows.
def odd():
    """Sizes that are no multiples of anything, GQA, dim != vdim, a layer that does not mix values before the first that
    does, a layer without a feed-forward, windows and caps per layer, one layer without a window."""
    return config([layer(6, 2, 12, 20, window=9, cap=7.0, v_mix=False, ff=36),
                   layer(6, 3, 20, 12, window=0, cap=0.0, v_mix=True, mlp=None),
                   layer(3, 3, 28, 12, window=17, cap=11.0, v_mix=True, mlp="moe", ff=20, experts=5, identity=2, top=3),
                   layer(9, 3, 12, 12, window=1, cap=3.0, v_mix=True, mlp="moe", ff=12, experts=7, identity=0, top=1,
                         groups=7, keep=3)], width=50, vocab=77, eps=3e-4)


def mixed():
    """Expert groups, identity experts, one key/value head per query head."""
    return config([layer(4, 4, 32, 32, window=21, mlp="moe", ff=24, experts=9, identity=6, top=4, groups=5, keep=2),
                   layer(4, 4, 32, 32, window=21, ff=72),
                   layer(4, 4, 32, 32, window=40, mlp="moe", ff=40, experts=8, identity=8, top=5, groups=2, keep=1)],
                  width=64, vocab=130)


def wide():
    """Head dims of the tensor-core attention's larger tile, several query heads per key/value head."""
    return config([layer(4, 1, 128, 128, window=130, cap=30.0, ff=200),
                   layer(8, 2, 96, 64, window=64, cap=60.0, v_mix=False, mlp="moe", ff=72, experts=6, identity=3, top=2,
                         groups=3, keep=2)], width=264, vocab=301)


CONFIGS = {"odd": odd, "mixed": mixed, "wide": wide}
