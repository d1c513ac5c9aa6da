"""Architectures.  Importing this package registers them."""
from . import bedenex, fivedra, llama, redarax, vufolorn, zonidra  # noqa: F401
