"""Sozanex model family (model.py: configuration, weights, state; step.py: the step function)."""
from .model import Sozanex, SozanexArgs, sozanex_configs  # noqa: F401
