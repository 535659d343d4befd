"""Architectures: each module turns its configuration into a ModelSpec and registers itself."""
from . import gpt2, mamusun, muzozen, nipolorn, podenex, sosutar, vipolix  # noqa: F401
