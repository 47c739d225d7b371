"""Futezen: registration of the architecture name with its configuration and model.  The model is the generic
``DecoderModel`` over ``FutezenConfig.model_spec()``: layers in the sandwich arrangement (a norm on both sides of every
sublayer), attention over a cached latent with low-rank queries, grouped-query attention or a state-space recurrence,
a dense gated feed-forward or routed experts beside a gated shared one, a stretch of layers that may run several
times, a final norm and the embedding table as the head."""
from __future__ import annotations

from ..config.futezen import FutezenConfig
from ..config.registry import register_architecture
from ..parts.base import Precision
from ..parts.model import DecoderModel


class FutezenForCausalLM(DecoderModel):
    config_class = FutezenConfig

    def __init__(self, config: FutezenConfig, precision: Precision, device):
        self.config = config
        super().__init__(config.model_spec(), precision, device)


register_architecture("Futezen", FutezenConfig, FutezenForCausalLM)
