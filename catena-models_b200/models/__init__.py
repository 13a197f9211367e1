"""Architectures.  Importing this package registers them by name."""
from . import fozedra, kofadra, lfm3, maferax, narasun, relilix  # noqa: F401
