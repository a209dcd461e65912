"""Architectures: each module registers its name, configuration class and builder."""
from . import bolelix, gesuvik, kamosun, lopazen, musavik, qwen3, susalorn  # noqa: F401
