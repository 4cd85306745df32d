"""llvq_b200: language models on NVIDIA B200 (sm_100a) — fused Leech-lattice dequant-GEMV weights, and dense bf16/f32
weights with latent attention."""
from ._lib import LlvqError, PUBLISHED_FINGERPRINT  # noqa: F401
from .registry import load_model  # noqa: F401
from .runtime import FusedProj, FusedRuntime  # noqa: F401

__all__ = ["FusedRuntime", "FusedProj", "LlvqError", "PUBLISHED_FINGERPRINT", "load_model"]
