"""Built-in architectures. Importing this package registers them."""
from . import bubalix, delunex, linurax, luzitar, pilonex, qwen3, rolevik  # noqa: F401
