"""tensorwarp_b200 — LLM inference kernels and engines for NVIDIA B200.

``csrc/`` holds the sm_100a kernels of two libraries: the TW-Marlin W4A16 Q4 GEMM family and its decode
step (``include/twmarlin.h``, ``include/twm_decode.h``; host mirror in ``quantize`` and ``generate``),
and decoder models with dense 16-bit or 32-bit weights (``include/twm_dense.h``; ``dense``, ``engine``).
``registry`` loads a model by its configuration, ``scheduler`` serves requests on it.  Importing the
package does not load a library; the first call does, and fails loudly if it cannot.
"""
from . import _lib  # noqa: F401
from .build import build  # noqa: F401

__all__ = ["build", "quantize", "registry"]
