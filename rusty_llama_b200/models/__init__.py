"""Architectures.  Importing this package registers them."""

from . import damadra, fakelorn, llama, namalix, revirax, tefavik, vezatar  # noqa: F401
