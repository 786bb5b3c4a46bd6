"""Built-in architectures.  Importing this package registers them."""
from . import beputar, ginodra, kilisun, muvonex, nomudra, qwen3, vozorax  # noqa: F401
