"""Architectures.  Importing this package registers each of them by name."""
from . import bikovik, bisudra, fasesun, nugolorn, pegurax, qwen3, tukulorn  # noqa: F401
