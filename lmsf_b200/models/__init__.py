"""Architectures.  Importing this package registers them."""
from . import bedenex, dizepel, fivedra, llama, redarax, vufolorn, zonidra  # noqa: F401
