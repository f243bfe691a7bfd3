"""Decoders the paged engine serves, by family name (``checkpoint.safetensors_io.FAMILIES``
maps a checkpoint's architecture to one): how a family reads its configuration and builds its
model.  ``serve``, ``keep`` and the trace replay all go through this table."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Optional

import torch


@dataclass(frozen=True)
class PagedDecoder:
    config: Callable                     # parsed config.json -> configuration object
    named_config: Callable               # "tiny" or None (the default shape) -> configuration
    model: Callable                      # (configuration, device, dtype, ctx) -> model, no weights
    gpu_dtypes: tuple                    # types the family's GPU path runs in
    build_group: Optional[str] = None    # build.GROUPS entry that suffices for this family


def _qwen3_config(d):
    from .qwen3_moe import Qwen3MoeConfig
    return Qwen3MoeConfig.from_hf(d)


def _qwen3_named(name):
    from .qwen3_moe import Qwen3MoeConfig
    return Qwen3MoeConfig.tiny() if name == "tiny" else Qwen3MoeConfig.qwen3_30b_a3b()


def _qwen3_model(cfg, device, dtype, ctx=None):
    from .qwen3_moe import Qwen3MoeModel
    return Qwen3MoeModel(cfg, device, dtype, ctx)


def _nepevik_config(d):
    from .nepevik import NepevikConfig
    return NepevikConfig.from_json(d)


def _nepevik_named(name):
    from .nepevik import NepevikConfig
    return NepevikConfig.tiny() if name == "tiny" else NepevikConfig.bench()


def _nepevik_model(cfg, device, dtype, ctx=None):
    from .nepevik import NepevikModel
    if ctx is not None and ctx.world_size > 1:
        raise ValueError("this family is served on one GPU")
    return NepevikModel(cfg, device, dtype)


def _zonopel_config(d):
    from .zonopel import ZonopelConfig
    return ZonopelConfig.from_json(d)


def _zonopel_named(name):
    from .zonopel import ZonopelConfig
    return ZonopelConfig.tiny() if name == "tiny" else ZonopelConfig.bench()


def _zonopel_model(cfg, device, dtype, ctx=None):
    from .zonopel import ZonopelModel
    if ctx is not None and ctx.world_size > 1:
        raise ValueError("this family is served on one GPU")
    return ZonopelModel(cfg, device, dtype)


def _tadinex_config(d):
    from .tadinex import TadinexConfig
    return TadinexConfig.from_json(d)


def _tadinex_named(name):
    from .tadinex import TadinexConfig
    return TadinexConfig.tiny() if name == "tiny" else TadinexConfig.bench()


def _tadinex_model(cfg, device, dtype, ctx=None):
    from .tadinex import TadinexModel
    if ctx is not None and ctx.world_size > 1:
        raise ValueError("this family is served on one GPU")
    return TadinexModel(cfg, device, dtype)


def _nopuzen_config(d):
    from .nopuzen import NopuzenConfig
    return NopuzenConfig.from_json(d)


def _nopuzen_named(name):
    from .nopuzen import NopuzenConfig
    return NopuzenConfig.tiny() if name == "tiny" else NopuzenConfig.bench()


def _nopuzen_model(cfg, device, dtype, ctx=None):
    from .nopuzen import NopuzenModel
    if ctx is not None and ctx.world_size > 1:
        raise ValueError("this family is served on one GPU")
    return NopuzenModel(cfg, device, dtype)


PAGED_DECODERS = {
    "qwen3_moe": PagedDecoder(_qwen3_config, _qwen3_named, _qwen3_model, (torch.bfloat16,)),
    "nepevik": PagedDecoder(_nepevik_config, _nepevik_named, _nepevik_model,
                            (torch.bfloat16, torch.float32), "nepevik"),
    "zonopel": PagedDecoder(_zonopel_config, _zonopel_named, _zonopel_model,
                            (torch.bfloat16, torch.float32), "zonopel"),
    "tadinex": PagedDecoder(_tadinex_config, _tadinex_named, _tadinex_model,
                            (torch.bfloat16, torch.float32), "tadinex"),
    "nopuzen": PagedDecoder(_nopuzen_config, _nopuzen_named, _nopuzen_model,
                            (torch.bfloat16, torch.float32), "nopuzen"),
}


def named_family(model: str) -> Optional[str]:
    """Paged decoder that a model name without a checkpoint (``random:<family>[:tiny]``) names."""
    return next((f for f in PAGED_DECODERS if f in model.lower()), None)
