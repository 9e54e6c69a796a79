"""Architecture recipes (registered on import) and the decoder they build."""

from . import fovudra, labolix, mekusun, qwen2, zelasun, zururax, zuzunex  # noqa: F401
from .decoder import DecoderModel, model_tensor_specs, slot_needs

__all__ = ["DecoderModel", "model_tensor_specs", "slot_needs"]
