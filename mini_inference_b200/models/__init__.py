"""Built-in architectures; importing this package registers them."""
from . import fetodra, kofutar, megovik, naditar, namesun, nununex, qwen3  # noqa: F401
