"""Architectures known to the registry; importing this package registers them."""

from . import bafavik, kivurax, parunex, qwen3, venarax, vesidra, zozezen  # noqa: F401
