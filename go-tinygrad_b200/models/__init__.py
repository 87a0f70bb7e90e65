"""Architectures the library ships with.  Importing this package registers them."""
from . import letanex, llama, megerax, mererax, ropovik, senupel, zotolix  # noqa: F401  (registration)
