"""Built-in architectures.  Importing this package registers them."""
from . import demavik, lizizen, mamivik, peratar, petanex, qwen2, redalix  # noqa: F401
