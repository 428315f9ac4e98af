"""Importing this package registers every architecture the engine ships."""

from . import bumalix, dogotar, gekopel, goganex, llama, nerenex, zomolix  # noqa: F401
