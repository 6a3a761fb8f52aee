"""Architectures: each module turns its typed configuration into a ``ModelSpec`` and
registers itself by the name found in config.json."""
from . import fekolorn, kopatar, pozelix, pusazen, qwen3, rusadra, sumuvik

__all__ = ["fekolorn", "kopatar", "pozelix", "pusazen", "qwen3", "rusadra", "sumuvik"]
