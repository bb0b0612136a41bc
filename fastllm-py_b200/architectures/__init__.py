"""Importing this package registers the architectures the engine ships with."""
from . import kerirax, lasonex, llama, lufozen, saberax, sakusun, tigitar  # noqa: F401
