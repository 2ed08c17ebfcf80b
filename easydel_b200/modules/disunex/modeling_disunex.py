"""Disunex: a decoder of latent-attention layers (sliding window, a sink per head, output gate) with dense or expert
feed-forwards, each branch followed by a norm of the weighted sum, over a residual stream kept in 32 bits. A layer may
use the weights of another one with a cache of its own.

The family is a mapping: the configuration lists every layer with its own sizes, and this module turns that list into
the spec-driven decoder's fields (:class:`..._base.decoder.ArchSpec`) and the checkpoint's tensor names into module names.
The mechanisms live beside their kin: ``layers/mla.py`` (:class:`LatentStreamAttention`) over ``ops/latent.py``,
``layers/moe.py`` (sigmoid scores with a correction, clamped gated units), ``ops/stream.py`` (norm after the sum).
"""

from __future__ import annotations

import torch

from ...infra.base_config import EasyDeLBaseConfig
from ...infra.factory import TaskType, register_config, register_module
from .._base.decoder import ArchSpec, DecoderForCausalLM, DecoderModel, MoESpec


def _default_layers(width: int) -> list[dict]:
    mixer = {"heads": 16, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256, "scale": 96 ** -0.5,
             "rot": {"base": 10000.0, "dims": 32}, "mask": {"size": 1024}}
    return [{"type": "latent_attention", "mixer": mixer, "mlp": {"kind": "dense", "ff": 4 * width}},
            {"type": "latent_attention", "mixer": mixer,
             "mlp": {"kind": "moe", "router": {"experts": 32, "top": 4}, "expert": {"ff": width, "limit": 7.0}}}]


@register_config("disunex", architecture="Disunex")
class DisunexConfig(EasyDeLBaseConfig):
    """``layers``: one entry per layer run, ``{"type": "latent_attention", "mixer": {sizes}, "mlp": {"kind": "dense", "ff"}
    | {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff", "limit"}} | None, "weights_of": j (optional)}``;
    ``norm``: ``{"eps"}``; ``postln_alpha``: weight of the stream in every sum; ``vocab``; ``width``."""

    model_type = "disunex"
    hf_config_keys = ("layers", "norm", "postln_alpha", "vocab", "width")

    def __init__(self, layers=None, norm=None, postln_alpha=1.0, vocab=32000, width=1024, architecture="Disunex",
                 max_position_embeddings=131072, initializer_range=0.02, tie_word_embeddings=True, **kw):
        self.layers = list(_default_layers(width) if layers is None else layers)
        self.norm, self.postln_alpha = dict(norm or {"eps": 1e-6}), postln_alpha
        self.vocab, self.width = vocab, width
        self.architecture = architecture
        self.max_position_embeddings, self.initializer_range = max_position_embeddings, initializer_range
        for i, layer in enumerate(self.layers):
            if layer["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            mlp = layer.get("mlp")
            if mlp is not None and mlp["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            if mlp is not None and mlp["kind"] == "moe" and not 1 <= mlp["router"]["top"] <= mlp["router"]["experts"]:
                raise ValueError(f"layer {i}: {mlp['router']['top']} of {mlp['router']['experts']} experts")
            if layer.get("weights_of") is not None and not 0 <= layer["weights_of"] < len(self.layers):
                raise ValueError(f"layer {i} uses the weights of layer {layer['weights_of']}, which does not exist")
        self.weight_layers()
        super().__init__(tie_word_embeddings=tie_word_embeddings, **kw)

    def weight_layers(self) -> tuple[list[int], list[int]]:
        """(entries that own weights, in order; for every entry, which of those it uses)."""
        owner = []
        for i, layer in enumerate(self.layers):
            j, seen = i, set()
            while self.layers[j].get("weights_of") is not None:
                if j in seen:
                    raise ValueError(f"layer {i}: its weights are nobody's own")
                seen.add(j)
                j = self.layers[j]["weights_of"]
            owner.append(j)
        own = sorted(set(owner))
        return own, [own.index(j) for j in owner]

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
        return max(m["mixer"]["heads"] for m in self.layers)

    @property
    def head_dim(self) -> int:
        return max(m["mixer"]["dim"] + m["mixer"]["rot_dim"] for m in self.layers)


def _layer_fields(entry: dict) -> dict:
    """Overrides of the :class:`ArchSpec` fields for one layer entry."""
    m, mlp = entry["mixer"], entry.get("mlp")
    rot = m["rot"]
    out = {"num_heads": m["heads"], "intermediate_size": 0, "moe": None,
           "mla": {"dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"],
                   "scale": m["scale"], "rope_base": rot["base"], "rope_dims": rot["dims"],
                   "sliding_window": (m.get("mask") or {}).get("size"), "use_sinks": True, "output_gate": True}}
    if mlp is not None and mlp["kind"] == "dense":
        out["intermediate_size"] = mlp["ff"]
    elif mlp is not None:
        out["moe"] = MoESpec(num_experts=mlp["router"]["experts"], top_k=mlp["router"]["top"],
                             intermediate_size=mlp["expert"]["ff"], scoring="sigmoid", use_score_bias=True,
                             expert_limit=mlp["expert"]["limit"], expert_init_std=0.02)
    return out


def disunex_spec(c: DisunexConfig) -> ArchSpec:
    own, runs = c.weight_layers()
    fields = tuple(_layer_fields(c.layers[j]) for j in own)
    return ArchSpec(hidden_size=c.width, num_layers=len(own), vocab_size=c.vocab, num_kv_heads=1,
                    head_dim=c.head_dim, num_heads=fields[0]["num_heads"], intermediate_size=0, mla=fields[0]["mla"],
                    max_position=c.max_position_embeddings, norm_eps=c.norm["eps"], norm_offset=1.0, act="gelu",
                    mlp="plain", pos_emb="none", residual="post_sum", residual_alpha=float(c.postln_alpha),
                    residual_f32=True, layer_runs=tuple(runs), per_layer=fields, init_std=c.initializer_range,
                    tie_embeddings=True)


#: checkpoint name -> module name, for the part after ``l<i>.`` and for the whole name outside the layers
_LAYER_NAMES = {
    "norm1": "post_attention_layernorm.weight", "norm2": "post_feedforward_layernorm.weight",
    "mix.q": "self_attn.q_proj.weight", "mix.dkv": "self_attn.dkv_proj.weight", "mix.g": "self_attn.g_proj.weight",
    "mix.dkv.norm": "self_attn.kv_norm.weight", "mix.uk": "self_attn.uk_proj.weight",
    "mix.uv": "self_attn.uv_proj.weight", "mix.sink": "self_attn.sinks", "mix.o": "self_attn.o_proj.weight",
}
_DENSE_NAMES = {"mlp.up": "mlp.fc1.weight", "mlp.down": "mlp.fc2.weight"}
_MOE_NAMES = {"mlp.router": "mlp.gate.weight", "mlp.correction": "mlp.e_score_correction_bias"}
_TOP_NAMES = {"embed": "embed_tokens.weight", "final.norm": "norm.weight"}


def _names_of(config: DisunexConfig, prefix: str) -> dict[str, str]:
    """The whole checkpoint-to-module name table of one configuration; entries that use another layer's weights have no
    names of their own."""
    out = {k: prefix + v for k, v in _TOP_NAMES.items()}
    for i, j in enumerate(config.weight_layers()[0]):
        mlp, names = config.layers[j].get("mlp"), dict(_LAYER_NAMES)
        if mlp is None:
            names.pop("norm2")
        elif mlp["kind"] == "dense":
            names.update(_DENSE_NAMES)
        else:
            names.update(_MOE_NAMES)
            for e in range(mlp["router"]["experts"]):
                names.update({f"mlp.e{e}.{p}": f"mlp.experts.{e}.{p}_proj.weight" for p in ("gate", "up", "down")})
        out.update({f"l{j}.{k}": f"{prefix}layers.{i}.{v}" for k, v in names.items()})
    return out


class _DisunexNames:
    """Checkpoint naming hooks of the state-dict converter."""

    _name_prefix = "model."

    def hf_rename_in(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        table = _names_of(self.config, self._name_prefix)
        return {table.get(k, k): v for k, v in state.items()}

    def hf_rename_out(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        table = {v: k for k, v in _names_of(self.config, self._name_prefix).items()}
        return {table.get(k, k): v for k, v in state.items()}


@register_module(TaskType.BASE_MODULE, config=DisunexConfig, model_type="disunex")
class DisunexModel(_DisunexNames, DecoderModel):
    spec_fn = staticmethod(disunex_spec)
    _name_prefix = ""


@register_module(TaskType.CAUSAL_LM, config=DisunexConfig, model_type="disunex")
class DisunexForCausalLM(_DisunexNames, DecoderForCausalLM):
    backbone_cls = DisunexModel
