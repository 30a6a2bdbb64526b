"""Architectures the library knows.  Importing registers them."""
from . import kisilix, lenesun, lfm3, nolapel, tevilix, zafilix, zekivik  # noqa: F401
