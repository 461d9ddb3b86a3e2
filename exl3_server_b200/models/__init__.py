"""Architectures: each module turns its configuration into a plan and registers itself."""
from . import llama, nibelix, nikodra, potodra, rigitar, soporax, tunavik  # noqa: F401
