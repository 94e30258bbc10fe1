"""Rigalorn model family (model.py: configuration, weights, state; step.py: the step function)."""
from .model import Rigalorn, RigalornArgs, rigalorn_configs  # noqa: F401
