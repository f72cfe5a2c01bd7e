"""Architectures: each module registers its config parser and tensor naming."""
from . import kepusun, llama, lomopel, mobatar, runevik, tazulix, vuvalorn  # noqa: F401
