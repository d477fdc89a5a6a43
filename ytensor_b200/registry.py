"""Model registry: which class, weight file and compiled sources belong to the architecture a config.json names.

    model = load_model("folder", dtype="bfloat16", max_tokens=4096)     # config.json + weights
    tokens = model.generate_greedy(prompt_ids, 32)
"""
from __future__ import annotations

import json
from dataclasses import dataclass
from pathlib import Path
from typing import Callable

# sources (csrc/*.cu) every model is linked with
_CORE = ("runtime", "gemm", "flash_attn", "rowops", "sampling", "lm_rows")
_NATIVE = _CORE + ("moe", "lm_decode", "lm_model")


@dataclass(frozen=True)
class Model:
    name: str
    dtypes: tuple            # number formats the model runs in
    sources: tuple           # csrc/*.cu that hold its kernels
    load: Callable           # (folder, config dict, dtype, batch, max_tokens) -> CausalLM


def _native(config_class, model_class, folder: Path, config: dict, dtype: str, batch: int, max_tokens: int):
    from .safetensors import SafetensorsFile
    m = model_class(config_class.from_dict(config), batch=batch, max_tokens=max_tokens, dtype=dtype)
    m.load_weights(SafetensorsFile(folder / "model.safetensors"))
    return m


def _load_duzozen(*args):
    from .duzozen import DuzozenConfig, DuzozenForCausalLM
    return _native(DuzozenConfig, DuzozenForCausalLM, *args)


def _load_derupel(*args):
    from .derupel import DerupelConfig, DerupelForCausalLM
    return _native(DerupelConfig, DerupelForCausalLM, *args)


def _load_qwen3(folder: Path, config: dict, dtype: str, batch: int, max_tokens: int):
    from .qwen3 import Qwen3Config, Qwen3ForCausalLM
    from .ytfile import load_qwen3_checkpoint
    known = {k: config[k] for k in Qwen3Config.__dataclass_fields__ if k in config}
    known["max_position_embeddings"] = max_tokens
    cfg = Qwen3Config(**known)
    m = Qwen3ForCausalLM(cfg, batch=batch)
    m.load_weights(load_qwen3_checkpoint(folder / "model.yt", cfg))
    return m


MODELS = {
    "Duzozen": Model("Duzozen", ("bfloat16", "float32"), _NATIVE + ("duzozen",), _load_duzozen),
    "Derupel": Model("Derupel", ("bfloat16", "float32"), _NATIVE + ("latent_attn", "decayed_attn", "derupel"), _load_derupel),
    # (bf16 weights with fp32 activations: the one format it has)
    "Qwen3ForCausalLM": Model("Qwen3ForCausalLM", ("bfloat16",), _CORE + ("elementwise", "decoder"), _load_qwen3),
}


class UnsupportedModel(ValueError):
    pass


def read_config(folder) -> dict:
    return json.loads((Path(folder) / "config.json").read_text())


def find_model(config: dict) -> Model:
    """The registered model of a config.json: its "architecture", or the first known name of its "architectures"."""
    names = [config["architecture"]] if "architecture" in config else list(config.get("architectures", ()))
    for n in names:
        if n in MODELS:
            return MODELS[n]
    raise UnsupportedModel(f"no registered model for {names or 'a config.json without an architecture'}; "
                           f"known: {', '.join(sorted(MODELS))}")


def load_model(folder, dtype: str = "bfloat16", batch: int = 1, max_tokens: int = 4096, build: bool = False):
    """The model of `folder` with its weights on the current CUDA device. build: compile what the model needs first when
    the library is missing or out of date."""
    config = read_config(folder)
    entry = find_model(config)
    if dtype not in entry.dtypes:
        raise UnsupportedModel(f"{entry.name} does not run in {dtype}")
    if build:
        from . import _lib
        from .build import ensure
        _lib.full_library = False
        ensure(entry.sources)
    return entry.load(Path(folder), config, dtype, batch, max_tokens)
