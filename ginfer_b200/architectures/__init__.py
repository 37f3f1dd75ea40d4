"""Architectures known to the registry; importing this package registers them."""
from . import bapivik, daburax, lasizen, pimidra, qwen2, vilepel, zolapel  # noqa: F401
