"""Built-in architectures; importing this package registers them."""
from . import galupel, gevulorn, kuterax, logozen, pugadra, qwen3, tidenex  # noqa: F401
