"""Architectures.  Importing this package registers them."""
from . import dugulorn, givirax, legalix, lorulix, qwen3, rumurax, sumevik  # noqa: F401
