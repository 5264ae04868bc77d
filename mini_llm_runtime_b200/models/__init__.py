"""Importing this package registers the architectures."""
from . import gelulix, gopevik, niridra, qwen3, repolix, sokolorn, sopetar  # noqa: F401
