"""Architectures this engine builds.  Importing a module registers its architecture name."""
from . import bilolorn, desilorn, kusolorn, neburax, nugolorn, qwen3, zinunex  # noqa: F401
