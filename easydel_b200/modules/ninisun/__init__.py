"""Ninisun: windowed attention with kept first tokens and blended values, and sigmoid attention beside a generalised delta
rule, every branch normed and scaled before it joins the stream."""

from .modeling_ninisun import NinisunConfig, NinisunForCausalLM, NinisunModel

__all__ = ["NinisunConfig", "NinisunModel", "NinisunForCausalLM"]
