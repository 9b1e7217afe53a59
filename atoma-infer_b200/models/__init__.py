"""Architectures built from the parts; importing this package registers them."""
from . import bumolix, dosovik, kavotar, kulivik, llama, tupunex, tutezen  # noqa: F401
