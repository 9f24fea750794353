"""Architectures.  Importing this package registers them."""

from . import dopudra, fuzazen, gurolix, llama, pudulorn, zadurax  # noqa: F401
