"""Architectures.  Importing this package registers them."""

from . import fakelorn, llama, namalix, revirax, tefavik, vezatar  # noqa: F401
