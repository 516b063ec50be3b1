"""Built-in architectures.  Importing this package registers them."""
from . import gulipel, kakirax, malapel, qwen3, sakinex, sarizen, ziginex  # noqa: F401
