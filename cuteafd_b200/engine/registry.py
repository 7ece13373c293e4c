"""Model name or snapshot directory -> model description, device weights, engine: the one place that knows which engine runs which kind of
model on a single GPU (multi-GPU layouts build their rank engines in `parallel.runner`)."""
from __future__ import annotations

import dataclasses
import os

from ..config import NAMED_SPECS, ModelSpec, spec_by_name, spec_from_snapshot

DTYPES = {"bfloat16": "bf16", "float32": "f32"}


def model_spec(model: str, *, layers: int = 0, dtype: str = "bfloat16") -> ModelSpec:
    """`layers` > 0 keeps that many layers of a named shape; `dtype` "float32" runs everything in fp32 (layer stacks only)."""
    if model in NAMED_SPECS:
        spec = spec_by_name(model)
        if layers:
            spec = NAMED_SPECS[model](n_layers=layers) if spec.blocks else spec.replace(n_layers=layers)
    else:
        spec = spec_from_snapshot(model)
        if layers and not spec.blocks:
            spec = spec.replace(n_layers=layers)
    if dtype != "bfloat16":
        if dtype not in DTYPES:
            raise ValueError(f"dtype {dtype!r}: one of {sorted(DTYPES)}")
        if not spec.blocks:
            raise ValueError(f"{spec.name}: only layer stacks run in {dtype}")
        k = DTYPES[dtype]
        spec = spec.replace(quant=dataclasses.replace(spec.quant, dense=k, experts=k, kv=k))
    return spec


def load_weights(model: str, spec: ModelSpec, device, seed: int = 1):
    """Weights of a snapshot in the forms the kernels consume, or synthetic ones for a named shape."""
    from ..models.weights import DeviceWeights
    snapshot = os.path.isdir(model)
    if spec.stack == "mixed":
        from ..models.mixed_stack import mixed_weights_from_masters, mixed_weights_random
        if snapshot:
            from ..loader.stack_checkpoint import read_mixed_masters
            return mixed_weights_from_masters(spec, read_mixed_masters(model, spec), device)
        return mixed_weights_random(spec, device, seed=seed)
    if spec.stack == "hyper":
        from ..models.hyper_stack import hyper_weights_from_masters, hyper_weights_random
        if snapshot:
            from ..loader.stack_checkpoint import read_hyper_masters
            return hyper_weights_from_masters(spec, read_hyper_masters(model, spec), device)
        return hyper_weights_random(spec, device, seed=seed)
    if spec.stack == "hybrid":
        from ..models.hybrid_stack import hybrid_weights_from_masters, hybrid_weights_random
        if snapshot:
            from ..loader.stack_checkpoint import read_hybrid_masters
            return hybrid_weights_from_masters(spec, read_hybrid_masters(model, spec), device)
        return hybrid_weights_random(spec, device, seed=seed)
    if spec.blocks:
        from ..models.latent_stack import stack_weights_from_masters, stack_weights_random
        if snapshot:
            from ..loader.stack_checkpoint import read_stack_masters
            return stack_weights_from_masters(spec, read_stack_masters(model, spec), device)
        return stack_weights_random(spec, device, seed=seed)
    if spec.attn.kind == "mla":
        from .mla import mla_weights_from_masters, mla_weights_random
        if snapshot:
            from ..loader.checkpoint import read_masters
            return mla_weights_from_masters(spec, read_masters(model, spec), device)
        return mla_weights_random(spec, device, seed=seed)
    if snapshot:
        from ..loader.checkpoint import load_device_weights
        return load_device_weights(model, spec, device)         # tensors in their stored formats, no repacking
    if spec.name == "tiny":
        from ..ref.model import init_weights
        return DeviceWeights.from_masters(spec, init_weights(spec, 0), device)
    return DeviceWeights.random(spec, device, seed=seed)


def engine_class(spec: ModelSpec):
    if spec.stack == "mixed":
        from .mixed_stack import MixedStackEngine
        return MixedStackEngine
    if spec.stack == "hyper":
        from .hyper_stack import HyperStackEngine
        return HyperStackEngine
    if spec.stack == "hybrid":
        from .hybrid_stack import HybridStackEngine
        return HybridStackEngine
    if spec.blocks:
        from .latent_stack import LatentStackEngine
        return LatentStackEngine
    if spec.attn.kind == "mla":
        from .mla import MlaEngine
        return MlaEngine
    from .engine import Engine
    return Engine


def build_engine(spec: ModelSpec, weights, **kw):
    return engine_class(spec)(weights, **kw)
