"""Which class opens which model: the reference's list of factories whose TryCreate either accepts a model or passes
(NFAI.Models.Llama3/LlamaModelFactory.cs:36-44), extended to models that are described by a config.json.
"""
from __future__ import annotations

import json
import os
from typing import Callable, Dict, Optional

from .api import CausalModel, CudaContext, LlamaModel, ModelOptions, PlannedModel


def _open_gguf(ctx: CudaContext, options: ModelOptions) -> CausalModel:
    return LlamaModel.from_gguf_native(ctx, options.GGUFPath, options.KVCacheSize, options.KVCacheDType)


def _open_planned(ctx: CudaContext, options: ModelOptions) -> CausalModel:
    dtype = "bf16" if options.WeightDType == "auto" else options.WeightDType
    return PlannedModel(ctx, options.ModelPath, options.KVCacheSize, dtype)


# "architecture" of config.json -> how to open it
CONFIG_ARCHITECTURES: Dict[str, Callable[[CudaContext, ModelOptions], CausalModel]] = {"Tometar": _open_planned, "Tutizen": _open_planned}


def architecture_of(path: str) -> str:
    """The architecture a model folder names in its config.json."""
    with open(os.path.join(path, "config.json")) as fh:
        return str(json.load(fh).get("architecture", ""))


def try_create(ctx: CudaContext, options: ModelOptions) -> Optional[CausalModel]:
    """The model options.ModelPath (a folder) or options.GGUFPath names, or None if no class takes it."""
    if options.ModelPath:
        opener = CONFIG_ARCHITECTURES.get(architecture_of(options.ModelPath))
        return opener(ctx, options) if opener else None
    return _open_gguf(ctx, options)
