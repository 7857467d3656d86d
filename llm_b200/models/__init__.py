from . import fopivik, kepevik, llama, nidorax, norusun, potipel, tevudra  # noqa: F401  (each registers its architecture)
from .spec import LayerSpec, ModelSpec, PartSpec

__all__ = ["LayerSpec", "ModelSpec", "PartSpec"]
