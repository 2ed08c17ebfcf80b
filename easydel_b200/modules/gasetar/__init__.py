"""Gasetar: windowed attention with capped scores and latent attention with sinks and gates, beside feed-forwards that read
the same norm."""

from .modeling_gasetar import GasetarConfig, GasetarForCausalLM, GasetarModel

__all__ = ["GasetarConfig", "GasetarModel", "GasetarForCausalLM"]
