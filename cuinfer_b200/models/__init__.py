"""Architectures this engine builds.  Importing a module registers its architecture name."""
from . import bilolorn, desilorn, kusolorn, nugolorn, qwen3, zinunex  # noqa: F401
