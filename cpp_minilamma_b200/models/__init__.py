"""Architectures.  Importing the package registers them by their `architectures` name."""
from . import badolix, gopitar, kupirax, llama, malulorn, mefolorn, sopanex  # noqa: F401
