"""Model families: which reader, weight set and model class a checkpoint folder gets, decided by its
config.json. ``from_pretrained`` is what the command line, the examples and the trace runner use;
``register`` adds a family."""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable, List, Optional

import torch


@dataclass(frozen=True)
class ModelFamily:
    name: str
    matches: Callable[[dict], bool]            # config.json -> is it this family
    weights: Callable                          # (model_dir, config, device, dtype, layout) -> (weights, cfg)
    model: Callable                            # weights -> model
    kernels: str = "all"                       # kernel set that suffices when nothing is built yet (_build.SETS)


_FAMILIES: List[ModelFamily] = []


def register(family: ModelFamily) -> None:
    """Families registered later are asked first."""
    _FAMILIES.insert(0, family)


def families() -> List[str]:
    return [f.name for f in _FAMILIES]


def read_json(model_dir: str) -> dict:
    with open(os.path.join(model_dir, "config.json")) as f:
        return json.load(f)


def family_of(config: dict) -> ModelFamily:
    for f in _FAMILIES:
        if f.matches(config):
            return f
    raise ValueError(f"no model family for this config.json (architecture {config.get('architecture')!r}, "
                     f"model_type {config.get('model_type')!r}); known: {families()}")


def from_pretrained(model_dir: str, device="cuda", dtype: Optional[torch.dtype] = None):
    """The model of a checkpoint folder, ready for ``ServingEngine``."""
    config = read_json(model_dir)
    fam = family_of(config)
    if torch.device(device).type == "cuda":
        from .. import _lib
        _lib.prefer_kernels(fam.kernels)
    weights, _cfg = fam.weights(model_dir, config, device, dtype or torch.bfloat16, None)
    return fam.model(weights)


# ------------------------------------------------------------------------------------------------
def _transformer_weights(model_dir, config, device, dtype, layout):
    from ..loader import safetensors_loader as L
    cfg, quant = L.read_config(model_dir)
    return L.build_weights(cfg, L.load_tensors(model_dir), quant, device, dtype, layout), cfg


def _transformer_model(weights):
    from .mixtral import MixtralModel
    from .qwen import Qwen2Model
    from .transformer import TransformerModel
    cls = {"qwen2": Qwen2Model, "mixtral": MixtralModel}.get(weights.cfg.name, TransformerModel)
    return cls(weights)


def _posudra_weights(model_dir, config, device, dtype, layout):
    from ..config import PosudraConfig
    from ..loader.safetensors_loader import load_tensors
    from .posudra import build_weights
    if layout is not None and layout.world != 1:
        raise ValueError("Posudra runs on one GPU")
    cfg = PosudraConfig.from_json(config)
    return build_weights(cfg, load_tensors(model_dir), device, dtype), cfg


def _posudra_model(weights):
    from .posudra import PosudraModel
    return PosudraModel(weights)


def _rodapel_weights(model_dir, config, device, dtype, layout):
    from ..config import RodapelConfig
    from ..loader.safetensors_loader import load_tensors
    from .rodapel import build_weights
    if layout is not None and layout.world != 1:
        raise ValueError("Rodapel runs on one GPU")
    cfg = RodapelConfig.from_json(config)
    return build_weights(cfg, load_tensors(model_dir), device, dtype), cfg


def _rodapel_model(weights):
    from .rodapel import RodapelModel
    return RodapelModel(weights)


def _nugosun_weights(model_dir, config, device, dtype, layout):
    from ..config import NugosunConfig
    from ..loader.safetensors_loader import load_tensors
    from .nugosun import build_weights
    if layout is not None and layout.world != 1:
        raise ValueError("Nugosun runs on one GPU")
    cfg = NugosunConfig.from_json(config)
    return build_weights(cfg, load_tensors(model_dir), device, dtype), cfg


def _nugosun_model(weights):
    from .nugosun import NugosunModel
    return NugosunModel(weights)


def _nizorax_weights(model_dir, config, device, dtype, layout):
    from ..config import NizoraxConfig
    from ..loader.safetensors_loader import load_tensors
    from .nizorax import build_weights
    if layout is not None and layout.world != 1:
        raise ValueError("Nizorax runs on one GPU")
    cfg = NizoraxConfig.from_json(config)
    return build_weights(cfg, load_tensors(model_dir), device, dtype), cfg


def _nizorax_model(weights):
    from .nizorax import NizoraxModel
    return NizoraxModel(weights)


register(ModelFamily("transformer", lambda c: "num_attention_heads" in c, _transformer_weights, _transformer_model))
register(ModelFamily("posudra", lambda c: c.get("architecture") == "Posudra", _posudra_weights, _posudra_model,
                     kernels="parallel_block"))
register(ModelFamily("rodapel", lambda c: c.get("architecture") == "Rodapel", _rodapel_weights, _rodapel_model,
                     kernels="post_norm"))
register(ModelFamily("nugosun", lambda c: c.get("architecture") == "Nugosun", _nugosun_weights, _nugosun_model,
                     kernels="twin_norm"))
register(ModelFamily("nizorax", lambda c: c.get("architecture") == "Nizorax", _nizorax_weights, _nizorax_model,
                     kernels="sandwich"))
