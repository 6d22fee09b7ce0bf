"""Architectures this engine serves.  Importing the package registers them."""

from . import kavedra, nulazen, qwen2, radilix, sadodra, setotar, vupitar  # noqa: F401
