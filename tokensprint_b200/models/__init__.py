"""Architectures.  Importing this package registers them (config/registry.py)."""

from tokensprint_b200.models import dazilix, fegetar, mugulorn, pekunex, qwen3, vasosun, vepevik  # noqa: F401
