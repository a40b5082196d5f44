"""Architectures that are not described by :class:`~arctic_platform_b200.models.config.DecoderConfig`.

A checkpoint directory whose ``config.json`` has an ``architecture`` key names one of these.  An entry gives the
configuration class (``from_dict``, ``PRESETS``) and the model class -- both are imported on first use -- and the kernel
sources (``csrc/*.cu``) of its layers.  The model class implements the serving protocol of
:mod:`arctic_platform_b200.engine.stateful_sampler`.
"""
from __future__ import annotations

import importlib
from typing import Any, Dict, Tuple

_ARCHITECTURES: Dict[str, Tuple[str, str, str]] = {}        # architecture -> (module, config class, model class)
_KERNELS: Dict[str, Tuple[str, ...]] = {}


def register_architecture(name: str, module: str, config_class: str, model_class: str, kernels: Tuple[str, ...] = ()) -> None:
    _ARCHITECTURES[name] = (module, config_class, model_class)
    _KERNELS[name] = tuple(kernels)


register_architecture("Reninex", "arctic_platform_b200.models.reninex", "ReninexConfig", "ReninexLM",
                      ("serve_attention", "serve_attention_tc", "retention", "retention_mma"))
register_architecture("Rigulorn", "arctic_platform_b200.models.rigulorn", "RigulornConfig", "RigulornLM",
                      ("serve_streams", "serve_softmax", "serve_softmax_tc", "ssm", "ssm_mma"))
register_architecture("Titatar", "arctic_platform_b200.models.titatar", "TitatarConfig", "TitatarLM",
                      ("serve_residual", "serve_latent", "serve_moe", "serve_softmax", "serve_softmax_wide", "serve_flash_tc"))
register_architecture("Meronex", "arctic_platform_b200.models.meronex", "MeronexConfig", "MeronexLM",
                      ("serve_residual", "serve_moe", "serve_softmax", "serve_flash_tc", "ssm", "recurrent", "memory_mma", "delta_mma",
                       "time_mix_mma"))


def kernel_sources(architecture: str) -> Tuple[str, ...]:
    """Sources of the kernels of the architecture's own layers (without extension)."""
    return _KERNELS[architecture]


def architectures() -> Tuple[str, ...]:
    return tuple(sorted(_ARCHITECTURES))


def config_class(architecture: str):
    if architecture not in _ARCHITECTURES:
        raise ValueError(f"unknown architecture {architecture!r} (known: {list(architectures())})")
    module, cfg, _ = _ARCHITECTURES[architecture]
    return getattr(importlib.import_module(module), cfg)


def presets() -> Dict[str, Any]:
    out: Dict[str, Any] = {}
    for module, _, _ in _ARCHITECTURES.values():
        out.update(importlib.import_module(module).PRESETS)
    return out


def new_model(cfg, device, dtype):
    """An uninitialised model for ``cfg`` -- the class its architecture names, else the standard decoder."""
    arch = getattr(cfg, "architecture", None)
    if arch is None:
        from .decoder import DecoderLM
        return DecoderLM(cfg, device, dtype)
    module, _, model = _ARCHITECTURES[arch]
    return getattr(importlib.import_module(module), model)(cfg, device, dtype)


def is_stateful(cfg) -> bool:
    """Whether the model is served by the stateful paged engine (and by nothing else in this package)."""
    return getattr(cfg, "architecture", None) is not None
