"""Architectures the engine can build.  Importing this package registers them."""
from . import lanirax, lunerax, munizen, pugozen, qwen3, rapovik, vamadra  # noqa: F401
