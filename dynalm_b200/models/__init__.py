"""Architectures; importing this package registers them."""
from . import bugapel, llama, nisotar, rematar, rodelorn, sipelorn, todupel  # noqa: F401
