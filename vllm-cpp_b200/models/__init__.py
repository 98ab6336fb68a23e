"""Architectures known to the registry."""
from . import gipinex, kasuvik, lutodra, qwen2, retodra, rolesun, rufisun  # noqa: F401
