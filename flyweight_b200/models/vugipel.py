"""Vugipel: registration of the architecture name with its configuration and model.  The model is the generic
``DecoderModel`` over ``VugipelConfig.model_spec()``: pre-norm layers (weights stored around zero) whose mixer is
a minGRU or a windowed attention with kept first tokens and rotated values beside a retention, experts behind a
sigmoid router whose scores weigh the experts' inputs, a final norm and an untied head."""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.vugipel import VugipelConfig
from ..parts.base import Precision
from ..parts.model import DecoderModel


class VugipelForCausalLM(DecoderModel):
    config_class = VugipelConfig

    def __init__(self, config: VugipelConfig, precision: Precision, device):
        self.config = config
        super().__init__(config.model_spec(), precision, device)


register_architecture("Vugipel", VugipelConfig, VugipelForCausalLM)
