"""Small Varolorn configurations with seeded weights, written as model folders, and the helpers that run them through
the engine and through the plain implementation.

The configurations differ from one another in every size and option: 1, 2, 3 and 5 query heads per key/value head and as many
as heads; values wider, narrower and as wide as keys; stretches shorter than a page, longer than one, of a page exactly, and
no mask at all; 2 to 24 distance buckets (odd counts among them) with largest distances below and above the stretch; values
mixed in every attention layer, in some and in none, with other layers in between; recurrences with one head and several,
one group, several and as many as heads, one norm part and several, one to five taps; feed-forwards and none; one, two, three
and five streams and plain residual sums; with and without pair rows (with one bucket, with more buckets than pairs, with
multipliers that overflow 32 bits); widths that are multiples of 64 and widths that no vectorised kernel takes; attention
heads that the bfloat16 kernels take as they are, padded to 64 and padded to 128.  Weights are N(0, 1/inputs) ("loud": every
layer changes the streams by as much as they hold)."""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

import plain_varolorn as P


def _att(heads, kv_heads, dim, vdim, scale, bias_max, size=0, v_mix=False, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_max": bias_max, "v_mix": v_mix}
    if size:
        m["mask"] = {"size": size}
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _ssm(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv,
                                        "norm_groups": norm_groups}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def _cfg(vocab, width, eps, layers, streams=None, scale=None, bigram=None):
    d = {"architecture": "Varolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if streams is not None:
        d["streams"] = streams
    emb = {}
    if scale is not None:
        emb["scale"] = scale
    if bigram is not None:
        emb["bigram"] = {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}
    if emb:
        d["embedding"] = emb
    return d


CONFIGS = {
    # three streams; values mixed past a layer of another kind and past one that does not mix; stretches shorter than a page
    "va": _cfg(101, 48, 1e-6, [_att(4, 2, 16, 12, 0.3, 9.5, size=7, v_mix=True, ff=40), _ssm(3, 10, 8, 1, 3, 2, ff=24),
                               _att(6, 2, 8, 12, 0.4, 30, size=21, v_mix=True), _att(2, 2, 12, 20, 0.25, 40, size=50),
                               _att(2, 2, 20, 12, 0.2, 100, size=33, v_mix=True, ff=16)], streams=3, scale=2.5, bigram=(37, 5, 11)),
    # one stream, no mask, no embedding section at all, a recurrence first and last
    "vb": _cfg(130, 64, 1e-5, [_ssm(4, 16, 16, 4, 4, 4), _att(8, 8, 8, 16, 0.35, 24, ff=72), _ssm(2, 24, 12, 2, 2, 1, ff=32)], streams=1),
    # sizes in multiples of 64 (what the tensor-core kernels take), five streams, multipliers beyond 32 bits
    "vc": _cfg(512, 128, 1e-5, [_att(8, 2, 64, 64, 0.12, 50, size=80, v_mix=True, ff=128), _ssm(4, 32, 64, 2, 4, 4, ff=64),
                                _att(6, 2, 64, 64, 0.15, 200, size=128, v_mix=True, ff=64), _att(4, 4, 64, 64, 0.11, 33, ff=128),
                                _ssm(8, 16, 32, 1, 5, 2)], streams=5, scale=1.5, bigram=(1000, 2147483659, 40503)),
    # the least there can be: one recurrence with one head and one tap on plain residual sums; one bucket of pairs
    "vd": _cfg(50, 32, 1e-5, [_ssm(1, 20, 4, 1, 1, 1)], scale=0.7, bigram=(1, 3, 7)),
    # sizes no vectorised kernel takes, five heads on one; two streams
    "ve": _cfg(71, 38, 1e-4, [_att(5, 1, 10, 7, 0.3, 13, size=5, v_mix=True, ff=10), _ssm(5, 3, 7, 5, 3, 5, ff=22),
                              _att(5, 1, 6, 7, 0.4, 17, size=40, v_mix=True)], streams=2, scale=3.0, bigram=(9973, 70, 1)),
    # heads padded to 64 and to 128 in bfloat16, the same values mixed across both; plain residual sums
    "vf": _cfg(256, 96, 1e-5, [_att(4, 2, 24, 40, 0.2, 60, size=100, v_mix=True, ff=48), _att(6, 2, 72, 40, 0.12, 90, size=70, v_mix=True),
                               _ssm(3, 32, 16, 3, 4, 1, ff=80), _att(2, 2, 128, 128, 0.1, 40, size=64, ff=32),
                               _att(16, 2, 64, 32, 0.14, 300, size=150)], scale=1.0, bigram=(300, 17, 4)),
}
REL_ROWS = {"va": (6, 5, 8, 24), "vb": (16,), "vc": (32, 12, 7), "vd": (), "ve": (2, 9), "vf": (10, 20, 3, 16)}


def bf16_round(a: np.ndarray) -> np.ndarray:
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy()


def make_weights(name: str, seed: int) -> dict[str, np.ndarray]:
    """Seeded weights that bfloat16 holds exactly, as float32, by tensor name."""
    import zinfer_b200 as z
    from zinfer_b200.config.registry import build_model

    cfg = CONFIGS[name]
    rng = np.random.default_rng(seed)
    model = build_model(z.config_from_dict(cfg))
    rel_rows = iter(REL_ROWS[name])
    W = {}
    for key, spec in model.weight_specs().items():
        shape = spec.shape
        last = key.split(".")[-1]
        if last == "rel":
            W[key] = rng.normal(0, 1.0, (next(rel_rows), shape[1]))
        elif last == "vmix":
            W[key] = rng.uniform(0.2, 0.8, shape)
        elif last == "b":
            W[key] = rng.normal(0, 0.3, shape)
        elif last == "dt_bias":
            W[key] = rng.normal(-1.0, 1.0, shape)
        elif last == "A_log":
            W[key] = rng.uniform(-4.0, 1.0, shape)
        elif last == "D" or key.endswith(("q.norm", "k.norm", "mix.norm")):
            W[key] = 1.0 + rng.normal(0, 0.3, shape)
        elif last in ("norm1", "norm2") or key == "final.norm":
            W[key] = rng.normal(0, 0.3, shape)                      # stored around zero
        elif ".hc" in key and last == "mix":
            W[key] = np.eye(shape[0]) + rng.normal(0, 0.3, shape)
        elif ".hc" in key:
            W[key] = rng.normal(0.7, 0.4, shape)
        elif last == "conv":
            W[key] = rng.normal(0, shape[-1] ** -0.5, shape)
        elif key in ("embed", "bigram"):
            W[key] = rng.normal(0, 0.6, shape)
        else:
            W[key] = rng.normal(0, shape[-1] ** -0.5, shape)
        W[key] = bf16_round(W[key])
    return W


def write_folder(folder, cfg: dict, W: dict[str, np.ndarray]) -> Path:
    from zinfer_b200.weights import write_safetensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {n: torch.from_numpy(np.asarray(a)).to(torch.bfloat16) for n, a in W.items()})
    return folder


def plain_logits(cfg: dict, W: dict[str, np.ndarray], tokens) -> np.ndarray:
    return P.forward(cfg, {n: a.astype(np.float64) for n, a in W.items()}, list(tokens))


def tokens_for(cfg: dict, seed: int, n: int) -> list[int]:
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


TOL = {"float32": 5e-5, "bfloat16": 4e-2}


def rel_err(got, ref) -> float:
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    scale = float(np.abs(ref).max())
    assert scale > 0 and got.shape == ref.shape, (got.shape, ref.shape)
    return float(np.abs(got - ref).max()) / scale
