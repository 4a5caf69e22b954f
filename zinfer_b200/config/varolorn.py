"""Typed configuration of the Varolorn architecture, read from its own config.json keys.

The file is nested: `vocab`, `width`, `norm.eps`, `embedding` {scale (the token rows are multiplied by it; 1 if absent),
bigram {buckets, mul_prev, mul_cur}}, `streams` (residual streams; absent = plain residual sums) and `layers`, a list with
one entry per layer:

* `type` "attention": `mixer` {heads, kv_heads, dim, vdim, scale, bias_max, mask {size}, v_mix}: grouped-query softmax
  attention without a rotation, with biases in its projections, normed query and key heads, a learned number per (distance
  bucket, head) on the scores (buckets up to the distance `bias_max`; how many is the tensor's own), queries that see only
  their own stretch of `mask.size` positions, a gate per head; with `v_mix` the layer's values are mixed with those of the
  first such layer;
* `type` "mamba2": `mixer` {heads, vdim, state, groups, conv, norm_groups}: the Mamba-2 recurrence (heads of vdim values and
  `state` channels, `groups` shared key/query groups, a convolution of `conv` taps, a norm in `norm_groups` parts);
* `mlp`: null or {kind "dense", ff}.

Every size and constant comes from here; what the file does not mention (no `bigram`, no `mask`, no `streams`) the model
does not have.  The design sets no longest sequence; `max_positions`, if a file has it, is only the default context
of an engine (else DEFAULT_CONTEXT)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Optional

from .base import ConfigError, ModelConfig, as_float, as_int, need

MIXER_TYPES = ("attention", "mamba2")
DEFAULT_CONTEXT = 8192


@dataclass(frozen=True)
class VarolornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    bias_max: float
    chunk: int = 0                      # 0 = every earlier token
    v_mix: bool = False


@dataclass(frozen=True)
class VarolornMamba2:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class VarolornLayer:
    type: str
    mixer: VarolornAttention | VarolornMamba2
    ff: Optional[int]                   # hidden units of the feed-forward, None = no feed-forward


@dataclass(frozen=True)
class VarolornBigram:
    buckets: int
    mul_prev: int
    mul_cur: int


def _obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if v is None:
        return {}
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: '{where}{key}' must be an object")
    return v


def _mixer(kind: str, m: dict, w: str):
    heads = as_int(m, w + "heads", need(m, "heads"), 1)
    vdim = as_int(m, w + "vdim", need(m, "vdim"), 1)
    if kind == "mamba2":
        return VarolornMamba2(heads, vdim, as_int(m, w + "state", need(m, "state"), 1), as_int(m, w + "groups", m.get("groups", 1), 1),
                              as_int(m, w + "conv", need(m, "conv"), 1), as_int(m, w + "norm_groups", m.get("norm_groups", 1), 1))
    mask = _obj(m, "mask", w)
    v_mix = m.get("v_mix", False)
    if not isinstance(v_mix, bool):
        raise ConfigError(f"config.json: '{w}v_mix' must be true or false, found {v_mix!r}")
    return VarolornAttention(heads, as_int(m, w + "kv_heads", m.get("kv_heads", heads), 1), as_int(m, w + "dim", need(m, "dim"), 1), vdim,
                             as_float(w + "scale", need(m, "scale")), as_float(w + "bias_max", need(m, "bias_max")),
                             chunk=as_int(mask, w + "mask.size", need(mask, "size"), 1) if mask else 0, v_mix=v_mix)


def _ff(ml, w: str) -> Optional[int]:
    if ml is None:
        return None
    if not isinstance(ml, dict):
        raise ConfigError(f"config.json: '{w}' must be an object or null")
    if ml.get("kind", "dense") != "dense":
        raise ConfigError(f"config.json: '{w}.kind' = {ml['kind']!r}; the one known kind is 'dense'")
    return as_int(ml, w + ".ff", need(ml, "ff"), 1)


@dataclass
class VarolornConfig(ModelConfig):
    layers: tuple[VarolornLayer, ...] = ()
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    bigram: Optional[VarolornBigram] = None
    streams: int = 0                    # 0 = plain residual sums

    @classmethod
    def from_json_dict(cls, d: dict[str, Any]) -> "VarolornConfig":
        vocab = as_int(d, "vocab", need(d, "vocab"), 1)
        width = as_int(d, "width", need(d, "width"), 1)
        norm, emb = _obj(d, "norm", ""), _obj(d, "embedding", "")
        bg = _obj(emb, "bigram", "embedding.")
        bigram = None
        if bg:
            w = "embedding.bigram."
            bigram = VarolornBigram(as_int(bg, w + "buckets", need(bg, "buckets"), 1), as_int(bg, w + "mul_prev", need(bg, "mul_prev")),
                                    as_int(bg, w + "mul_cur", need(bg, "mul_cur")))
        raw_layers = need(d, "layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: 'layers[{i}]' must be an object")
            kind = str(need(L, "type"))
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: 'layers[{i}].type' = {kind!r}; known types are {list(MIXER_TYPES)}")
            layers.append(VarolornLayer(kind, _mixer(kind, _obj(L, "mixer", f"layers[{i}]."), f"layers[{i}].mixer."),
                                        _ff(L.get("mlp"), f"layers[{i}].mlp")))
        eos = d.get("eos_token_id")
        max_pos = d.get("max_positions")
        cfg = cls(architecture=str(d.get("architecture") or (d.get("architectures") or ["Varolorn"])[0]),
                  vocab_size=vocab, hidden_size=width,
                  max_position_embeddings=DEFAULT_CONTEXT if max_pos is None else as_int(d, "max_positions", max_pos, 1),
                  eos_token_ids=() if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos])),
                  raw=dict(d), layers=tuple(layers), norm_eps=as_float("norm.eps", norm.get("eps", 1e-5)),
                  embedding_scale=as_float("embedding.scale", emb.get("scale", 1.0)), bigram=bigram,
                  streams=0 if d.get("streams") is None else as_int(d, "streams", d["streams"], 1))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.norm_eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, found {self.norm_eps}")
        first = None
        for i, L in enumerate(self.layers):
            m, w = L.mixer, f"config.json: layers[{i}]"
            if L.type == "mamba2":
                if m.heads % m.groups:
                    raise ConfigError(f"{w}: {m.heads} heads are not a multiple of {m.groups} groups")
                if (m.heads * m.vdim) % m.norm_groups:
                    raise ConfigError(f"{w}: {m.heads * m.vdim} values cannot be normalised in {m.norm_groups} equal parts")
                continue
            if m.heads % m.kv_heads:
                raise ConfigError(f"{w}: {m.heads} heads are not a multiple of {m.kv_heads} kv_heads")
            if m.bias_max <= 1:
                raise ConfigError(f"{w}.mixer.bias_max must be above 1, found {m.bias_max}")
            if m.v_mix:
                first = m if first is None else first
                if (m.kv_heads, m.vdim) != (first.kv_heads, first.vdim):
                    raise ConfigError(f"{w}: layers that mix values need the first such layer's kv_heads and vdim")

    def first_value_layer(self) -> Optional[int]:
        """The first layer whose values the later `v_mix` layers mix into theirs."""
        return next((i for i, L in enumerate(self.layers) if L.type == "attention" and L.mixer.v_mix), None)

    def to_json_dict(self) -> dict[str, Any]:
        layers = []
        for L in self.layers:
            m = L.mixer
            if L.type == "mamba2":
                mixer: dict[str, Any] = {"heads": m.heads, "vdim": m.vdim, "state": m.state, "groups": m.groups, "conv": m.conv,
                                         "norm_groups": m.norm_groups}
            else:
                mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale,
                         "bias_max": m.bias_max, "v_mix": m.v_mix}
                if m.chunk:
                    mixer["mask"] = {"size": m.chunk}
            layers.append({"type": L.type, "mixer": mixer, "mlp": None if L.ff is None else {"kind": "dense", "ff": L.ff}})
        emb: dict[str, Any] = {"scale": self.embedding_scale}
        if self.bigram is not None:
            emb["bigram"] = {"buckets": self.bigram.buckets, "mul_prev": self.bigram.mul_prev, "mul_cur": self.bigram.mul_cur}
        d: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "embedding": emb, "layers": layers}
        if self.streams:
            d["streams"] = self.streams
        if self.max_position_embeddings != DEFAULT_CONTEXT:
            d["max_positions"] = self.max_position_embeddings
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
