"""Disunex: windowed latent attention with gates and sinks, norms after the sum, dense and expert feed-forwards, layers
that are used more than once."""

from .modeling_disunex import DisunexConfig, DisunexForCausalLM, DisunexModel

__all__ = ["DisunexConfig", "DisunexModel", "DisunexForCausalLM"]
