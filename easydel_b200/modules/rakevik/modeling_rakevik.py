"""Rakevik: a decoder whose layers are HGRN2 or softmax-attention mixers in any order, each with a token shift and an
optional xIELU feed-forward, over a residual stream kept in 32 bits; a range of layers runs several times in a row.

The family is a mapping: the configuration lists every layer with its own sizes, and this module turns that list into
the spec-driven decoder's fields (:class:`..._base.decoder.ArchSpec`) and the checkpoint's tensor names into module names.
The mechanisms live beside their kin: ``layers/hgrn2.py``, ``layers/attention.py`` (value size of its own, sinks,
per-head norms, query temperature), ``layers/mlp.py`` (xIELU), ``ops/stream.py`` (norm + token shift), and the loop in
``modules/_base/decoder.py``.
"""

from __future__ import annotations

import torch

from ...infra.base_config import EasyDeLBaseConfig
from ...infra.factory import TaskType, register_config, register_module
from .._base.decoder import ArchSpec, DecoderForCausalLM, DecoderModel

@register_config("rakevik", architecture="Rakevik")
class RakevikConfig(EasyDeLBaseConfig):
    """``layers``: one entry per layer, ``{"type": "hgrn2" | "attention", "mixer": {sizes}, "mlp": {"kind": "dense",
    "ff": n} | None}``; ``loop``: ``{"start", "stop", "times"}`` or None; ``norm``: ``{"eps"}``; ``vocab``; ``width``."""

    model_type = "rakevik"
    hf_config_keys = ("layers", "loop", "norm", "vocab", "width")

    def __init__(self, layers=None, loop=None, norm=None, vocab=32000, width=1024, architecture="Rakevik",
                 max_position_embeddings=131072, initializer_range=0.02, tie_word_embeddings=False, **kw):
        if layers is None:
            mlp = {"kind": "dense", "ff": 4 * width}
            layers = [{"type": "hgrn2", "mixer": {"heads": 8, "dim": 128, "vdim": 128}, "mlp": mlp},
                      {"type": "attention", "mixer": {"heads": 8, "kv_heads": 8, "dim": 128, "vdim": 128,
                                                      "scale": 128 ** -0.5}, "mlp": mlp}]
        self.layers, self.loop, self.norm = list(layers), loop, dict(norm or {"eps": 1e-6})
        self.vocab, self.width = vocab, width
        self.architecture = architecture
        self.max_position_embeddings, self.initializer_range = max_position_embeddings, initializer_range
        for i, layer in enumerate(self.layers):
            if layer["type"] not in ("hgrn2", "attention"):
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            m = layer["mixer"]
            if layer["type"] == "attention" and m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key/value heads")
        if loop is not None and not 0 <= loop["start"] <= loop["stop"] <= len(self.layers):
            raise ValueError(f"loop {loop} does not fit {len(self.layers)} layers")
        super().__init__(tie_word_embeddings=tie_word_embeddings, **kw)

    # the names the rest of the framework reads
    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def vocab_size(self) -> int:
        return self.vocab

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def num_attention_heads(self) -> int:
        return max((m["mixer"]["heads"] for m in self.layers if m["type"] == "attention"), default=1)

    @property
    def head_dim(self) -> int:
        return max((m["mixer"]["dim"] for m in self.layers if m["type"] == "attention"), default=1)


def _layer_fields(entry: dict) -> dict:
    """Overrides of the :class:`ArchSpec` fields for one layer entry."""
    m, mlp = entry["mixer"], entry.get("mlp")
    out = {"intermediate_size": mlp["ff"] if mlp else 0}
    if entry["type"] == "hgrn2":
        out["hgrn2"] = {"heads": m["heads"], "dim": m["dim"], "vdim": m["vdim"]}
        return out
    temp = m.get("q_temp")
    out.update(num_heads=m["heads"], num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"],
               attn_scale=m["scale"], attn_temp_tuning=(temp["coef"], temp["every"]) if temp else None)
    return out


def rakevik_spec(c: RakevikConfig) -> ArchSpec:
    first = next((_layer_fields(e) for e in c.layers if e["type"] == "attention"), None)
    base = {"num_heads": 1, "num_kv_heads": 1, "head_dim": 64} if first is None else \
        {k: first[k] for k in ("num_heads", "num_kv_heads", "head_dim", "v_head_dim")}
    loop = (c.loop["start"], c.loop["stop"], c.loop["times"]) if c.loop else None
    return ArchSpec(hidden_size=c.width, num_layers=len(c.layers), intermediate_size=0, vocab_size=c.vocab, **base,
                    max_position=c.max_position_embeddings, norm_eps=c.norm["eps"], act="xielu", mlp="plain",
                    qk_norm="rms_head", pos_emb="none", use_sinks=True, residual_f32=True, token_shift=True, loop=loop,
                    layer_types=tuple("hgrn2" if e["type"] == "hgrn2" else "full" for e in c.layers),
                    per_layer=tuple(_layer_fields(e) for e in c.layers), init_std=c.initializer_range,
                    tie_embeddings=False)


#: checkpoint name -> module name, for the part after ``l<i>.`` and for the whole name outside the layers
_LAYER_NAMES = {
    "norm1": "input_layernorm.weight", "norm2": "post_attention_layernorm.weight", "shift": "shift",
    "mlp.up": "mlp.fc1.weight", "mlp.down": "mlp.fc2.weight", "mlp.act": "mlp.act_params",
}
_MIXER_NAMES = {
    "attention": {"q": "self_attn.q_proj.weight", "k": "self_attn.k_proj.weight", "v": "self_attn.v_proj.weight",
                  "q.norm": "self_attn.q_norm.weight", "k.norm": "self_attn.k_norm.weight", "sink": "self_attn.sinks",
                  "o": "self_attn.o_proj.weight"},
    "hgrn2": {"q": "linear_attn.q_proj.weight", "f": "linear_attn.f_proj.weight", "v": "linear_attn.v_proj.weight",
              "f.b": "linear_attn.f_bias", "lower": "linear_attn.lower", "norm": "linear_attn.norm.weight",
              "o": "linear_attn.o_proj.weight"},
}
_TOP_NAMES = {"embed": "embed_tokens.weight", "loop.in": "loop_in.weight", "loop.step": "loop_step",
              "final.norm": "norm.weight"}


def _names_of(config: RakevikConfig, prefix: str) -> dict[str, str]:
    """The whole checkpoint-to-module name table of one configuration."""
    out = {k: prefix + v for k, v in _TOP_NAMES.items()}
    for i, entry in enumerate(config.layers):
        for k, v in _LAYER_NAMES.items():
            out[f"l{i}.{k}"] = f"{prefix}layers.{i}.{v}"
        for k, v in _MIXER_NAMES[entry["type"]].items():
            out[f"l{i}.mix.{k}"] = f"{prefix}layers.{i}.{v}"
    out["head"] = "lm_head.weight"
    return out


class _RakevikNames:
    """Checkpoint naming hooks of the state-dict converter."""

    _name_prefix = "model."

    def hf_rename_in(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        table = _names_of(self.config, self._name_prefix)
        return {table.get(k, k): v for k, v in state.items()}

    def hf_rename_out(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        table = {v: k for k, v in _names_of(self.config, self._name_prefix).items()}
        return {table.get(k, k): v for k, v in state.items()}


@register_module(TaskType.BASE_MODULE, config=RakevikConfig, model_type="rakevik")
class RakevikModel(_RakevikNames, DecoderModel):
    spec_fn = staticmethod(rakevik_spec)
    _name_prefix = ""


@register_module(TaskType.CAUSAL_LM, config=RakevikConfig, model_type="rakevik")
class RakevikForCausalLM(_RakevikNames, DecoderForCausalLM):
    backbone_cls = RakevikModel
