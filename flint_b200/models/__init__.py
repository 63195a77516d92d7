"""Architectures.  Importing this package registers the built-in ones."""
from . import dumizen, gepadra, phimoe, puledra, sinilorn, sokipel, tefovik  # noqa: F401
