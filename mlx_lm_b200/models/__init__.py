"""Architectures that ship with the package; importing this package registers them."""
from . import dalorax, fisesun, gpt2, lelatar, nufetar, vobusun, zuluvik  # noqa: F401
