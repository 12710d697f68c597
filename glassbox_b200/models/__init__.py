"""Architectures. Importing this package registers them."""
from . import babotar, felovik, llama, lodenex, lonorax, tagenex, zurerax  # noqa: F401
