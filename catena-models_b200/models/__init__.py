"""Architectures.  Importing this package registers them by name."""
from . import fozedra, kofadra, lfm3, maferax, mogilorn, narasun, relilix  # noqa: F401
