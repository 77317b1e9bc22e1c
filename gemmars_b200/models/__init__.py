"""Architectures.  Importing this package registers each of them under its config.json names."""
from . import dalerax, fezozen, kuporax, mevuvik, nogosun, qwen3, toretar  # noqa: F401
