"""Architectures.  Importing this package registers every architecture it holds."""

from . import gulazen, kudazen, nazulorn, nifalorn, paditar, qwen3, siparax  # noqa: F401
