"""Designs without a library implementation (``architecture`` instead of ``model_type`` in config.json), served by the hybrid
executor's stream layout in bf16 or fp32. Each module ``models/<name>.py`` has ``build_ / load_ / random_<name>_weights``,
``random_<name>_tensors`` and ``save_<name>_checkpoint``."""
from __future__ import annotations

from importlib import import_module

DESIGNS = ("fusolix", "govopel", "pamasun", "vavadra")


def design_fn(name: str, form: str):
    """``design_fn("pamasun", "load_{}_weights")``."""
    return getattr(import_module(f".{name}", __package__), form.format(name))
