"""Ketolix causal LM: the model class the registry hands out for ``"architecture": "Ketolix"`` (sublayers on the stream itself with a
norm on the way back; capped windowed attention with mixed values, convolved attention beside linear attention, matrix memory; tied
logits; `config.KetolixConfig`)."""
from __future__ import annotations

from ..config import KetolixConfig
from .hybrid import HybridForCausalLM


class KetolixForCausalLM(HybridForCausalLM):
    config_class = KetolixConfig
