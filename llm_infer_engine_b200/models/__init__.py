from . import burinex, dofipel, ganupel, llama, rogizen, selinex, zemivik  # noqa: F401  (register the architectures)
from .decoder import DecoderModel

__all__ = ["DecoderModel"]
