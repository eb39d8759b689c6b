"""Built-in architectures; importing this package registers them."""
from . import kutepel, llama, nemasun, rupotar, tokovik, vikarax, vonulorn  # noqa: F401
