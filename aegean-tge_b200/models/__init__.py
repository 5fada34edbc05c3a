"""Model assembly.  Importing this package registers the architectures it holds."""
from . import fesorax, kokolorn, lepizen, mozepel, puputar, qwen2, tazizen  # noqa: F401  (registration)
from .decoder import DecoderModel

__all__ = ["DecoderModel"]
