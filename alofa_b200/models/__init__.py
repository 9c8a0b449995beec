"""Built-in architectures.  Importing this package registers them."""
from . import darolix, dibulix, kikerax, kotutar, nugopel, pekerax, qwen2  # noqa: F401
