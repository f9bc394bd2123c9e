"""Architectures.  Importing this package registers the built-in ones."""
from . import buborax, fupapel, gpt2, lubavik, tukavik, zadunex, zuretar  # noqa: F401
