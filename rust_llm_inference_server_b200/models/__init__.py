"""Architectures known to the registry.  Importing the package registers them."""

from . import dotivik, gavodra, lanirax, lasapel, llama, papulix, rumedra  # noqa: F401
from .model import Model, build_model, load_model
