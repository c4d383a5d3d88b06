"""Architectures known to the registry.  Importing this package registers them."""
from . import dumalix, fofapel, fugavik, llama, salepel, tubazen, zufadra  # noqa: F401
