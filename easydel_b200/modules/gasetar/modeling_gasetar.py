"""Gasetar: a decoder of sliding-window attention layers (norms over the whole query and key projections, rotated halves
with scaled frequencies, capped scores) and latent attention layers (a sink per head, output gate) in any order, each
beside a dense or expert feed-forward that reads the same norm, over a residual stream kept in 32 bits.

The family is a mapping: the configuration lists every layer with its own sizes, and this module turns that list into
the spec-driven decoder's fields (:class:`..._base.decoder.ArchSpec`) and the checkpoint's tensor names into module names.
The mechanisms live beside their kin: ``layers/attention.py`` (full-width norms, rotation and soft-cap on the stream),
``layers/mla.py`` (:class:`LatentStreamAttention` with rotated halves), ``layers/moe.py`` (softmax over the chosen logits,
shared expert), ``ops/rotation.py``, ``ops/stream.py`` (sum of the branches and the next norm in one pass).
"""

from __future__ import annotations

import torch

from ...infra.base_config import EasyDeLBaseConfig
from ...infra.factory import TaskType, register_config, register_module
from .._base.decoder import ArchSpec, DecoderForCausalLM, DecoderModel, MoESpec


def _default_layers(width: int) -> list[dict]:
    windowed = {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0,
                "mask": {"size": 1024}, "rot": {"base": 10000.0, "dims": 128}}
    latent = {"heads": 16, "dim": 64, "rot_dim": 32, "vdim": 64, "kv_rank": 256, "scale": 96 ** -0.5,
              "rot": {"base": 10000.0, "dims": 32}}
    moe = {"kind": "moe", "router": {"experts": 32, "top": 4}, "expert": {"ff": width}, "shared": {"ff": width}}
    return [{"type": "attention", "mixer": windowed, "mlp": {"kind": "dense", "ff": 4 * width}},
            {"type": "latent_attention", "mixer": latent, "mlp": moe}]


@register_config("gasetar", architecture="Gasetar")
class GasetarConfig(EasyDeLBaseConfig):
    """``layers``: one entry per layer, ``{"type": "attention" | "latent_attention", "mixer": {sizes}, "mlp": {"kind":
    "dense", "ff"} | {"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}, "shared": {"ff"}} | None}``;
    ``embedding``: ``{"scale"}``; ``norm``: ``{"eps"}``; ``residual_mult``: factor of every layer's branches;
    ``logit_scale``, ``logit_softcap``; ``vocab``; ``width``."""

    model_type = "gasetar"
    hf_config_keys = ("layers", "embedding", "norm", "residual_mult", "logit_scale", "logit_softcap", "vocab", "width")

    def __init__(self, layers=None, embedding=None, norm=None, residual_mult=1.0, logit_scale=1.0, logit_softcap=0.0,
                 vocab=32000, width=1024, architecture="Gasetar", max_position_embeddings=131072, initializer_range=0.02,
                 tie_word_embeddings=True, **kw):
        self.layers = list(_default_layers(width) if layers is None else layers)
        self.embedding, self.norm = dict(embedding or {"scale": 1.0}), dict(norm or {"eps": 1e-6})
        self.residual_mult, self.logit_scale, self.logit_softcap = residual_mult, logit_scale, logit_softcap
        self.vocab, self.width = vocab, width
        self.architecture = architecture
        self.max_position_embeddings, self.initializer_range = max_position_embeddings, initializer_range
        for i, layer in enumerate(self.layers):
            if layer["type"] not in ("attention", "latent_attention"):
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            m, mlp = layer["mixer"], layer.get("mlp")
            if layer["type"] == "attention" and m["heads"] % m["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key/value heads")
            if mlp is not None and mlp["kind"] not in ("dense", "moe"):
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            if mlp is not None and mlp["kind"] == "moe" and not 1 <= mlp["router"]["top"] <= mlp["router"]["experts"]:
                raise ValueError(f"layer {i}: {mlp['router']['top']} of {mlp['router']['experts']} experts")
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
        return max(e["mixer"]["heads"] for e in self.layers)

    @property
    def head_dim(self) -> int:
        return max(e["mixer"]["dim"] + e["mixer"].get("rot_dim", 0) for e in self.layers)


def _layer_fields(entry: dict) -> dict:
    """Overrides of the :class:`ArchSpec` fields for one layer entry."""
    m, mlp = entry["mixer"], entry.get("mlp")
    rot = m["rot"]
    out = {"num_heads": m["heads"], "intermediate_size": 0, "moe": None}
    if entry["type"] == "attention":
        out.update(num_kv_heads=m["kv_heads"], head_dim=m["dim"], v_head_dim=m["vdim"], attn_scale=m["scale"],
                   attn_softcap=float(m.get("softcap") or 0.0), sliding_window=(m.get("mask") or {}).get("size"),
                   stream_rope={"base": rot["base"], "dims": rot["dims"], "scaling": rot.get("scaling")})
    else:
        out["mla"] = {"dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"], "kv_rank": m["kv_rank"],
                      "scale": m["scale"], "rope_base": rot["base"], "rope_dims": rot["dims"],
                      "rope_scaling": rot.get("scaling"), "rope_layout": "halves", "use_sinks": True, "output_gate": True}
    if mlp is not None and mlp["kind"] == "dense":
        out["intermediate_size"] = mlp["ff"]
    elif mlp is not None:
        out["moe"] = MoESpec(num_experts=mlp["router"]["experts"], top_k=mlp["router"]["top"],
                             intermediate_size=mlp["expert"]["ff"], scoring="softmax", router_bias=True,
                             shared_intermediate_size=(mlp.get("shared") or {}).get("ff", 0), expert_init_std=0.02)
    return out


def gasetar_spec(c: GasetarConfig) -> ArchSpec:
    fields = tuple(_layer_fields(e) for e in c.layers)
    windowed = next((f for f in fields if "mla" not in f), None)
    base = {"num_kv_heads": 1, "head_dim": c.head_dim} if windowed is None else \
        {k: windowed[k] for k in ("num_kv_heads", "head_dim", "v_head_dim")}
    return ArchSpec(hidden_size=c.width, num_layers=len(c.layers), vocab_size=c.vocab, num_heads=fields[0]["num_heads"],
                    intermediate_size=0, **base, max_position=c.max_position_embeddings, norm_eps=c.norm["eps"], act="silu",
                    mlp="gated", qk_norm="rms_full", pos_emb="none", residual="parallel", residual_f32=True,
                    residual_multiplier=float(c.residual_mult), embed_scale=float(c.embedding["scale"]),
                    logit_scale=float(c.logit_scale), logit_softcap=float(c.logit_softcap or 0.0),
                    layer_types=tuple("sliding" if f.get("sliding_window") else "full" for f in fields),
                    per_layer=fields, init_std=c.initializer_range, tie_embeddings=True)


#: checkpoint name -> module name, for the part after ``l<i>.`` and for the whole name outside the layers
_MIXER_NAMES = {
    "attention": {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "q.norm": "q_norm.weight",
                  "k.norm": "k_norm.weight", "o": "o_proj.weight"},
    "latent_attention": {"q": "q_proj.weight", "dkv": "dkv_proj.weight", "g": "g_proj.weight",
                         "dkv.norm": "kv_norm.weight", "uk": "uk_proj.weight", "uv": "uv_proj.weight", "sink": "sinks",
                         "o": "o_proj.weight"},
}
_UNIT_PARTS = ("gate", "up", "down")
_TOP_NAMES = {"embed": "embed_tokens.weight", "final.norm": "norm.weight"}


def _names_of(config: GasetarConfig, prefix: str) -> dict[str, str]:
    """The whole checkpoint-to-module name table of one configuration."""
    out = {k: prefix + v for k, v in _TOP_NAMES.items()}
    for i, entry in enumerate(config.layers):
        names = {"norm1": "input_layernorm.weight",
                 **{f"mix.{k}": f"self_attn.{v}" for k, v in _MIXER_NAMES[entry["type"]].items()}}
        mlp = entry.get("mlp")
        units = {}                            # checkpoint prefix -> module of every gated unit of the feed-forward
        if mlp is not None and mlp["kind"] == "dense":
            units["mlp"] = "mlp"
        elif mlp is not None:
            names.update({"mlp.router": "mlp.gate.weight", "mlp.router.b": "mlp.gate.bias"})
            units = {f"mlp.e{e}": f"mlp.experts.{e}" for e in range(mlp["router"]["experts"])}
            if mlp.get("shared"):
                units["mlp.shared"] = "mlp.shared_experts"
        names.update({f"{k}.{p}": f"{v}.{p}_proj.weight" for k, v in units.items() for p in _UNIT_PARTS})
        out.update({f"l{i}.{k}": f"{prefix}layers.{i}.{v}" for k, v in names.items()})
    return out


class _GasetarNames:
    """Checkpoint naming hooks of the state-dict converter."""

    _name_prefix = "model."

    def hf_rename_in(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        table = _names_of(self.config, self._name_prefix)
        return {table.get(k, k): v for k, v in state.items()}

    def hf_rename_out(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        table = {v: k for k, v in _names_of(self.config, self._name_prefix).items()}
        return {table.get(k, k): v for k, v in state.items()}


@register_module(TaskType.BASE_MODULE, config=GasetarConfig, model_type="gasetar")
class GasetarModel(_GasetarNames, DecoderModel):
    spec_fn = staticmethod(gasetar_spec)
    _name_prefix = ""


@register_module(TaskType.CAUSAL_LM, config=GasetarConfig, model_type="gasetar")
class GasetarForCausalLM(_GasetarNames, DecoderForCausalLM):
    backbone_cls = GasetarModel
