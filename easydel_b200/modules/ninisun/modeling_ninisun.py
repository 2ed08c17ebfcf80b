"""Ninisun: a decoder of sliding-window attention layers (the first tokens stay visible, values blend with the first such
layer's) and layers of two mixers side by side (attention with sigmoid weights and a gate per head, and a generalised delta
rule) in any order, with gated feed-forwards or none; every branch is normed and scaled per channel before it joins a
residual stream kept in 32 bits.

The family is a mapping: the configuration lists every layer with its own sizes, and this module turns that list into
the spec-driven decoder's fields (:class:`..._base.decoder.ArchSpec`) and the checkpoint's tensor names into module names.
The mechanisms live beside their kin: ``layers/attention.py`` (kept first tokens, blended values, sigmoid weights),
``layers/delta_rule.py``, ``layers/twin.py`` (two mixers over one projection), ``ops/rotation.py`` (YaRN, neighbours),
``ops/stream.py`` (a normed branch joins the stream and the next norm reads it in one pass).
"""

from __future__ import annotations

import copy
import math

import torch

from ...infra.base_config import EasyDeLBaseConfig
from ...infra.factory import TaskType, register_config, register_module
from .._base.decoder import ArchSpec, DecoderForCausalLM, DecoderModel

#: strongest decay of a token in the delta rule is e^-DECAY_RATE; added to the squared length of its keys
DECAY_RATE, UNIT_EPS = math.exp(-0.5), 1e-6


def _default_layers(width: int) -> list[dict]:
    mlp = {"kind": "dense", "ff": 4 * width}
    windowed = {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "v_mix": True,
                "mask": {"size": 1024, "keep_first": 4}, "rot": {"base": 1e6, "dims": 128}}
    twin = {"left": {"heads": 8, "kv_heads": 2, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                     "rot": {"base": 5e5, "dims": 128}}, "left_scale": 1.0,
            "right": {"heads": 16, "dim": 64, "rank": 64}, "right_scale": 1.0}
    return [{"type": "attention", "mixer": windowed, "mlp": mlp}, {"type": "parallel", "mixer": twin, "mlp": mlp}]


def _check_heads(i: int, m: dict) -> None:
    if m["heads"] % m["kv_heads"]:
        raise ValueError(f"layer {i}: {m['heads']} query heads over {m['kv_heads']} key/value heads")


@register_config("ninisun", architecture="Ninisun")
class NinisunConfig(EasyDeLBaseConfig):
    """``layers``: one entry per layer, ``{"type": "attention" | "parallel", "mixer": {sizes}, "mlp": {"kind": "dense", "ff"} |
    None}``; ``norm``: ``{"eps"}``; ``vocab``; ``width``. The rank of the delta rule's decay (``right.rank``) may be left to
    the checkpoint's tensors."""

    model_type = "ninisun"
    hf_config_keys = ("layers", "norm", "vocab", "width")

    def __init__(self, layers=None, norm=None, vocab=32000, width=1024, architecture="Ninisun",
                 max_position_embeddings=131072, initializer_range=0.02, tie_word_embeddings=True, **kw):
        self.layers = list(_default_layers(width) if layers is None else layers)
        self.norm = dict(norm or {"eps": 1e-6})
        self.vocab, self.width = vocab, width
        self.architecture = architecture
        self.max_position_embeddings, self.initializer_range = max_position_embeddings, initializer_range
        for i, layer in enumerate(self.layers):
            if layer["type"] not in ("attention", "parallel"):
                raise ValueError(f"layer {i}: unknown mixer type {layer['type']!r}")
            _check_heads(i, layer["mixer"]["left"] if layer["type"] == "parallel" else layer["mixer"])
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        super().__init__(tie_word_embeddings=tie_word_embeddings, **kw)

    @staticmethod
    def complete_from_shapes(fields: dict, shapes: dict[str, tuple[int, ...]]) -> dict:
        """Fills in the decay ranks that a checkpoint's configuration leaves to its tensors."""
        fields = copy.deepcopy(fields)
        for i, layer in enumerate(fields.get("layers") or ()):
            w1 = shapes.get(f"l{i}.mix.right.w1")
            if layer["type"] == "parallel" and w1 is not None:
                layer["mixer"]["right"].setdefault("rank", w1[0])
        return fields

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

    def _attention(self) -> list[dict]:
        return [e["mixer"]["left"] if e["type"] == "parallel" else e["mixer"] for e in self.layers]

    @property
    def num_attention_heads(self) -> int:
        return max(m["heads"] for m in self._attention())

    @property
    def head_dim(self) -> int:
        return max(m["dim"] for m in self._attention())


def _layer_fields(entry: dict) -> dict:
    """Overrides of the :class:`ArchSpec` fields for one layer entry."""
    mlp, twin = entry.get("mlp"), entry["type"] == "parallel"
    m = entry["mixer"]["left"] if twin else entry["mixer"]
    mask, rot = m.get("mask") or {}, m.get("rot")
    out = {"num_heads": m["heads"], "num_kv_heads": m["kv_heads"], "head_dim": m["dim"], "v_head_dim": m["vdim"],
           "attn_scale": m["scale"], "intermediate_size": mlp["ff"] if mlp else 0, "sliding_window": mask.get("size"),
           "keep_first": int(mask.get("keep_first") or 0), "value_mix": bool(m.get("v_mix")),
           "stream_rope": None if not rot else {"base": rot["base"], "dims": rot["dims"], "scaling": rot.get("scaling"),
                                                "layout": "neighbours"}}
    if twin:
        right = entry["mixer"]["right"]
        out.update(attn_bias=True, attn_score_bias=True,
                   twin={"delta": {"heads": right["heads"], "dim": right["dim"], "rank": right.get("rank", right["dim"]),
                                   "rate": DECAY_RATE, "unit_eps": UNIT_EPS},
                         "scales": (entry["mixer"]["left_scale"], entry["mixer"]["right_scale"])})
    return out


def ninisun_spec(c: NinisunConfig) -> ArchSpec:
    fields = tuple(_layer_fields(e) for e in c.layers)
    return ArchSpec(hidden_size=c.width, num_layers=len(c.layers), vocab_size=c.vocab, intermediate_size=0,
                    **{k: fields[0][k] for k in ("num_heads", "num_kv_heads", "head_dim", "v_head_dim")},
                    max_position=c.max_position_embeddings, norm_eps=c.norm["eps"], act="gelu_tanh", mlp="gated",
                    pos_emb="none", residual="pre", residual_f32=True, sandwich_norm=True, layer_scale=True,
                    layer_types=tuple("twin" if "twin" in f else "sliding" if f["sliding_window"] else "full" for f in fields),
                    per_layer=fields, init_std=c.initializer_range, tie_embeddings=True)


#: checkpoint name -> module name, for the part after ``l<i>.`` and for the whole name outside the layers
_LAYER_NAMES = {"norm1": "input_layernorm.weight", "norm1b": "post_attn_out_layernorm.weight", "ls1": "mixer_scale"}
_MLP_NAMES = {"norm2": "pre_feedforward_layernorm.weight", "norm2b": "post_feedforward_layernorm.weight", "ls2": "mlp_scale",
              **{f"mlp.{p}": f"mlp.{p}_proj.weight" for p in ("gate", "up", "down")}}
_ATTENTION_NAMES = {**{f"mix.{k}": f"self_attn.{k}_proj.weight" for k in "qkvo"}, "mix.vmix": "self_attn.value_mix"}
_TWIN_NAMES = {
    **{f"mix.left.{k}": f"mixer.left_{k}_proj.weight" for k in "qkvg"}, "mix.left.pb": "mixer.left.score_bias",
    **{f"mix.right.{k}": f"mixer.right_{k}_proj.weight" for k in "rkvag"}, "mix.right.w1": "mixer.right_x_proj.weight",
    "mix.right.w2": "mixer.right.decay_up.weight", "mix.right.w0": "mixer.right.decay_bias",
    "mix.right.a.b": "mixer.right.rate_bias", "mix.right.norm": "mixer.right.norm.weight",
}
_TOP_NAMES = {"embed": "embed_tokens.weight", "final.norm": "norm.weight"}


def _names_of(config: NinisunConfig, prefix: str) -> dict[str, str]:
    """Checkpoint-to-module name table of one configuration (tensors that map one to one)."""
    out = {k: prefix + v for k, v in _TOP_NAMES.items()}
    for i, entry in enumerate(config.layers):
        names = {**_LAYER_NAMES, **(_ATTENTION_NAMES if entry["type"] == "attention" else _TWIN_NAMES),
                 **(_MLP_NAMES if entry.get("mlp") is not None else {})}
        out.update({f"l{i}.{k}": f"{prefix}layers.{i}.{v}" for k, v in names.items()})
    return out


def _joined_of(config: NinisunConfig, prefix: str):
    """Module tensors that are several checkpoint tensors in a row: ``(module name, checkpoint names, axis, widths)``."""
    for i, entry in enumerate(config.layers):
        if entry["type"] != "parallel":
            continue
        a, r, at = entry["mixer"]["left"], entry["mixer"]["right"], f"{prefix}layers.{i}.mixer"
        yield (f"{at}.o_proj.weight", [f"l{i}.mix.{s}.o" for s in ("left", "right")], 1,
               [a["heads"] * a["vdim"], r["heads"] * r["dim"]])
        yield (f"{at}.left.qkv_bias", [f"l{i}.mix.left.{k}.b" for k in "qkv"], 0,
               [a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]])


class _NinisunNames:
    """Checkpoint naming hooks of the state-dict converter."""

    _name_prefix = "model."

    def hf_rename_in(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        for name, parts, axis, _ in _joined_of(self.config, self._name_prefix):
            if all(p in state for p in parts):
                state[name] = torch.cat([state.pop(p) for p in parts], axis)
        table = _names_of(self.config, self._name_prefix)
        return {table.get(k, k): v for k, v in state.items()}

    def hf_rename_out(self, state: dict[str, torch.Tensor]) -> dict[str, torch.Tensor]:
        for name, parts, axis, widths in _joined_of(self.config, self._name_prefix):
            if name in state:
                state.update(zip(parts, (t.contiguous() for t in torch.split(state.pop(name), widths, axis))))
        table = {v: k for k, v in _names_of(self.config, self._name_prefix).items()}
        return {table.get(k, k): v for k, v in state.items()}


@register_module(TaskType.BASE_MODULE, config=NinisunConfig, model_type="ninisun")
class NinisunModel(_NinisunNames, DecoderModel):
    spec_fn = staticmethod(ninisun_spec)
    _name_prefix = ""


@register_module(TaskType.CAUSAL_LM, config=NinisunConfig, model_type="ninisun")
class NinisunForCausalLM(_NinisunNames, DecoderForCausalLM):
    backbone_cls = NinisunModel
