"""Architectures. Importing this package registers them."""
from . import babotar, felovik, llama, lonorax, tagenex, zurerax  # noqa: F401
