"""Architectures.  Importing this package registers them with `beglin_b200.config.registry`."""
from . import dinatar, fanitar, nadilorn, qwen2, sofudra, sukisun, tuzupel  # noqa: F401
