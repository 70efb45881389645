"""Model designs described by a list of layers (``ModelSpec.layer_specs``): the module of each architecture.

A module has ``expected_tensors(spec)`` and ``unused_tensors(spec)`` (checkpoint manifest), ``build_weights(spec, source)``,
``random_weights(spec, seed, device)`` and ``build_model(weights, settings, comm)``."""
from __future__ import annotations

import importlib

MODULES = {"duponex": "duponex", "rudorax": "rudorax", "kabavik": "kabavik", "bazulorn": "bazulorn"}


def design(arch: str):
    """The architecture's module, or None for the architectures with uniform layers."""
    name = MODULES.get(arch)
    return importlib.import_module(f"{__package__}.{name}") if name else None
