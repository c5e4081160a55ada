"""Architectures; importing this package registers them."""
from . import bugapel, llama, rematar, rodelorn, sipelorn, todupel  # noqa: F401
