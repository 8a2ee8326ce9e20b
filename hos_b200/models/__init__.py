"""Architectures.  Importing this package registers them."""
from . import fobilorn, gemma2, nuvivik, ravutar, satapel, tofodra, vagonex  # noqa: F401
