"""Typed configuration of the Nipizen architecture, read from its own config.json keys.

The file is nested: `vocab`, `width`, `norm.eps` (of the layer norms and of every RMS norm inside the mixers) and `layers`, a
list with one entry per layer:

* `type` "parallel": `mixer` {left, right, left_scale, right_scale}, two mixers side by side: `left` {heads, kv_heads, dim, vdim,
  scale, rot {base, dims, scaling {factor, original, fast, slow}}}: grouped-query softmax attention; `right` {heads, kv_heads,
  dim, vdim, conv}: the gated delta rule with short convolutions of `conv` taps;
* `type` "mlstm": `mixer` {heads, dim, vdim, gate_cap}: a matrix memory with exponential gates;
* `mlp`: null or {kind "moe", expert {ff}, router {experts, top}}.

Every size and constant comes from here, but for the inner widths of the delta rule's low-rank maps, which are the tensors'
own; what the file does not mention (no `scaling`, no `rot`, no `kv_heads`, no `vdim`, a scale of a side) is the plain form: no
scaling, no rotation, as many as `heads`, as wide as `dim`, 1.  The design sets no longest sequence; `max_positions`, if a file
has it, is only the default context of an engine (else DEFAULT_CONTEXT)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Optional

from .base import ConfigError, ModelConfig, as_float, as_int, need

MIXER_TYPES = ("parallel", "mlstm")
DEFAULT_CONTEXT = 8192


@dataclass(frozen=True)
class NipizenAttention:            # the left side of a pair
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_base: float = 0.0
    rot_dims: int = 0              # 0 = no rotation
    yarn: Optional[tuple[float, float, float, float]] = None      # factor, original, fast, slow


@dataclass(frozen=True)
class NipizenDelta:                # the right side of a pair
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class NipizenMLstm:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class NipizenMlp:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class NipizenLayer:
    type: str
    left: Optional[NipizenAttention] = None
    right: Optional[NipizenDelta] = None
    left_scale: float = 1.0
    right_scale: float = 1.0
    mlstm: Optional[NipizenMLstm] = None
    mlp: Optional[NipizenMlp] = None


def _obj(d: dict, key: str, where: str) -> dict:
    v = d.get(key)
    if v is None:
        return {}
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: '{where}{key}' must be an object")
    return v


def _sizes(m: dict, w: str) -> tuple[int, int, int, int]:
    heads = as_int(m, w + "heads", need(m, "heads"), 1)
    dim = as_int(m, w + "dim", need(m, "dim"), 1)
    kv = m.get("kv_heads")
    vdim = m.get("vdim")
    return (heads, heads if kv is None else as_int(m, w + "kv_heads", kv, 1), dim,
            dim if vdim is None else as_int(m, w + "vdim", vdim, 1))


def _left(m: dict, w: str) -> NipizenAttention:
    heads, kv_heads, dim, vdim = _sizes(m, w)
    rot = _obj(m, "rot", w)
    sc = _obj(rot, "scaling", w + "rot.")
    scale = m.get("scale")
    dims = rot.get("dims")
    return NipizenAttention(
        heads, kv_heads, dim, vdim, dim ** -0.5 if scale is None else as_float(w + "scale", scale),
        rot_base=as_float(w + "rot.base", need(rot, "base")) if rot else 0.0,
        rot_dims=(dim if dims is None else as_int(rot, w + "rot.dims", dims, 0)) if rot else 0,
        yarn=tuple(as_float(f"{w}rot.scaling.{k}", need(sc, k)) for k in ("factor", "original", "fast", "slow")) if sc else None)


def _right(m: dict, w: str) -> NipizenDelta:
    return NipizenDelta(*_sizes(m, w), conv=as_int(m, w + "conv", need(m, "conv"), 1))


def _mlp(ml, w: str) -> Optional[NipizenMlp]:
    if ml is None:
        return None
    if not isinstance(ml, dict):
        raise ConfigError(f"config.json: '{w}' must be an object or null")
    kind = str(ml.get("kind", "moe"))
    if kind != "moe":
        raise ConfigError(f"config.json: '{w}.kind' = {kind!r}; the design's feed-forward is 'moe'")
    ex, ro = _obj(ml, "expert", w + "."), _obj(ml, "router", w + ".")
    return NipizenMlp(as_int(ex, w + ".expert.ff", need(ex, "ff"), 1), as_int(ro, w + ".router.experts", need(ro, "experts"), 1),
                      as_int(ro, w + ".router.top", need(ro, "top"), 1))


@dataclass
class NipizenConfig(ModelConfig):
    layers: tuple[NipizenLayer, ...] = ()
    norm_eps: float = 1e-5

    @classmethod
    def from_json_dict(cls, d: dict[str, Any]) -> "NipizenConfig":
        vocab = as_int(d, "vocab", need(d, "vocab"), 1)
        width = as_int(d, "width", need(d, "width"), 1)
        norm = _obj(d, "norm", "")
        raw_layers = need(d, "layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, L in enumerate(raw_layers):
            if not isinstance(L, dict):
                raise ConfigError(f"config.json: 'layers[{i}]' must be an object")
            kind = str(need(L, "type"))
            w = f"layers[{i}].mixer."
            m = _obj(L, "mixer", f"layers[{i}].")
            mlp = _mlp(L.get("mlp"), f"layers[{i}].mlp")
            if kind == "parallel":
                for side in ("left", "right"):
                    if not _obj(m, side, w):
                        raise ConfigError(f"config.json: required key '{w}{side}' is missing")
                scales = [1.0 if m.get(k) is None else as_float(w + k, m[k]) for k in ("left_scale", "right_scale")]
                layers.append(NipizenLayer(kind, left=_left(_obj(m, "left", w), w + "left."),
                                           right=_right(_obj(m, "right", w), w + "right."), left_scale=scales[0],
                                           right_scale=scales[1], mlp=mlp))
            elif kind == "mlstm":
                heads, _, dim, vdim = _sizes(m, w)
                layers.append(NipizenLayer(kind, mlstm=NipizenMLstm(heads, dim, vdim, as_float(w + "gate_cap", need(m, "gate_cap"))),
                                           mlp=mlp))
            else:
                raise ConfigError(f"config.json: 'layers[{i}].type' = {kind!r}; known types are {list(MIXER_TYPES)}")
        eos = d.get("eos_token_id")
        max_pos = d.get("max_positions")
        cfg = cls(architecture=str(d.get("architecture") or (d.get("architectures") or ["Nipizen"])[0]),
                  vocab_size=vocab, hidden_size=width,
                  max_position_embeddings=DEFAULT_CONTEXT if max_pos is None else as_int(d, "max_positions", max_pos, 1),
                  eos_token_ids=() if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos])),
                  raw=dict(d), layers=tuple(layers), norm_eps=as_float("norm.eps", norm.get("eps", 1e-5)))
        cfg.validate()
        return cfg

    def validate(self) -> None:
        if self.norm_eps <= 0:
            raise ConfigError(f"config.json: norm.eps must be positive, found {self.norm_eps}")
        for i, L in enumerate(self.layers):
            w = f"config.json: layers[{i}]"
            if L.type == "parallel":
                a, r = L.left, L.right
                if a is None or r is None:
                    raise ConfigError(f"{w}.mixer needs 'left' and 'right'")
                for side, m in (("left", a), ("right", r)):
                    if m.heads % m.kv_heads:
                        raise ConfigError(f"{w}.mixer.{side}: {m.heads} heads are not a multiple of {m.kv_heads} kv_heads")
                if a.rot_dims % 2 or a.rot_dims > a.dim:
                    raise ConfigError(f"{w}.mixer.left.rot.dims = {a.rot_dims} must be even and at most dim {a.dim}")
                if a.rot_dims and a.rot_base <= 0:
                    raise ConfigError(f"{w}.mixer.left.rot.base must be positive, found {a.rot_base}")
                if a.yarn is not None and (a.rot_base <= 1 or min(a.yarn) <= 0):
                    raise ConfigError(f"{w}.mixer.left.rot.scaling: {a.yarn} must be positive numbers, with a base above 1")
                if r.conv < 1:
                    raise ConfigError(f"{w}.mixer.right.conv must be at least 1, found {r.conv}")
            elif L.type == "mlstm":
                if L.mlstm is None or L.mlstm.gate_cap <= 0:
                    raise ConfigError(f"{w}.mixer.gate_cap must be positive")
            else:
                raise ConfigError(f"{w}.type = {L.type!r}; known types are {list(MIXER_TYPES)}")
            if L.mlp is not None and not 0 < L.mlp.top <= L.mlp.experts:
                raise ConfigError(f"{w}.mlp.router: {L.mlp.top} experts per token out of {L.mlp.experts}")

    def to_json_dict(self) -> dict[str, Any]:
        layers = []
        for L in self.layers:
            if L.type == "mlstm":
                m = L.mlstm
                mixer: dict[str, Any] = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "gate_cap": m.gate_cap}
            else:
                a, r = L.left, L.right
                left: dict[str, Any] = {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale}
                if a.rot_dims:
                    left["rot"] = {"base": a.rot_base, "dims": a.rot_dims}
                    if a.yarn is not None:
                        left["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), a.yarn))
                mixer = {"left": left, "right": {"heads": r.heads, "kv_heads": r.kv_heads, "dim": r.dim, "vdim": r.vdim, "conv": r.conv},
                         "left_scale": L.left_scale, "right_scale": L.right_scale}
            mlp = None
            if L.mlp is not None:
                mlp = {"kind": "moe", "expert": {"ff": L.mlp.ff}, "router": {"experts": L.mlp.experts, "top": L.mlp.top}}
            layers.append({"type": L.type, "mixer": mixer, "mlp": mlp})
        d: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size,
                             "norm": {"eps": self.norm_eps}, "layers": layers}
        if self.max_position_embeddings != DEFAULT_CONTEXT:
            d["max_positions"] = self.max_position_embeddings
        if self.eos_token_ids:
            d["eos_token_id"] = list(self.eos_token_ids)
        return d
