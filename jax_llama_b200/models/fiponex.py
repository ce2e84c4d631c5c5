"""Fiponex causal LM: the model class the registry hands out for ``"architecture": "Fiponex"`` (sandwich blocks over a scaled embedding;
attention with position-dependent query temperature and channel gates, windowed latent attention, gated delta rule with one decay per
head; relu-gated layers and experts; `config.FiponexConfig`)."""
from __future__ import annotations

from ..config import FiponexConfig
from .hybrid import HybridForCausalLM


class FiponexForCausalLM(HybridForCausalLM):
    config_class = FiponexConfig
