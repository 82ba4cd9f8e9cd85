"""Architectures: import the built-in ones so that they are registered."""
from . import fegizen, mistral, nodepel, saropel, sisadra, tubepel, zedivik  # noqa: F401
from .decoder import DecoderModel  # noqa: F401
