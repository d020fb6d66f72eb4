"""Architectures: importing this package registers every one of them."""

from . import bunosun, llama, pakarax, puvirax, rerilorn, simetar, zemarax  # noqa: F401
