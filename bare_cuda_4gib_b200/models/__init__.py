"""Architectures.  Importing this package registers them."""

from . import dopudra, fuzazen, gurolix, llama, pudulorn, sizitar, zadurax  # noqa: F401
