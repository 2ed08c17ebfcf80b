"""Rakevik: HGRN2 and attention layers over an fp32 residual stream, with a looped block of layers."""

from .modeling_rakevik import RakevikConfig, RakevikForCausalLM, RakevikModel

__all__ = ["RakevikConfig", "RakevikModel", "RakevikForCausalLM"]
