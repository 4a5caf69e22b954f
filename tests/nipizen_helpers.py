"""Small Nipizen configurations with seeded weights, written as model folders, and the helpers that run them through the engine
and through the plain implementation.

The configurations differ from one another in every size and option: 1, 2, 3 and 5 heads per key/value head on either side of a
pair; values wider, narrower and as wide as keys; rotations over the whole head, a part and none, with scaled frequencies whose
blend lies inside the pairs, at their ends and in one pair, and without scaling; convolutions of 1 to 5 taps; inner widths of
the low-rank maps unequal, odd and larger than the heads; one and several memories in an mLSTM, low and high caps; one, some and
all experts per token, and layers with no feed-forward; scales of the two sides equal, unequal, negative and absent; widths that are
multiples of 64 and widths that no vectorised kernel takes.  Weights are N(0, 1/inputs) ("loud": every layer changes the
stream by as much as it holds); the decays lie between 0.3 and 0.999."""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

import plain_nipizen as P


def _rot(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


def _pair(left, right, mlp=None, scales=(1.0, 1.0)):
    heads, kv, dim, vdim, scale, rot = left
    m = {"left": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale},
         "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right)), "left_scale": scales[0], "right_scale": scales[1]}
    if rot is not None:
        m["left"]["rot"] = rot
    return {"type": "parallel", "mixer": m, "mlp": mlp}


def _mem(heads, dim, vdim, cap, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def _moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


CONFIGS = {
    # two query heads per key/value head on the left, shared q/k heads on the right, a partial scaled rotation, three layers of all kinds
    "na": {"architecture": "Nipizen", "vocab": 97, "width": 48, "norm": {"eps": 1e-5},
           "layers": [_pair((4, 2, 16, 12, 0.3, _rot(1000.0, 8, (4.0, 64, 8.0, 0.5))), (4, 2, 12, 10, 3), _moe(6, 2, 24), (0.7, 0.9)),
                      _mem(3, 8, 10, 5.0, _moe(4, 1, 20)),
                      _pair((2, 1, 20, 20, 0.2, _rot(100.0, 20)), (3, 3, 10, 14, 2), None, (1.2, -0.4))]},
    # every expert chosen (no choice to make), no rotation, one tap
    "nb": {"architecture": "Nipizen", "vocab": 130, "width": 64, "norm": {"eps": 1e-6},
           "layers": [_mem(2, 16, 8, 2.0, _moe(3, 3, 16)), _pair((6, 6, 8, 16, 0.35, None), (5, 1, 16, 24, 1), _moe(2, 2, 72), (0.5, 0.5))]},
    # sizes the tensor-core kernels take
    "nc": {"architecture": "Nipizen", "vocab": 384, "width": 192, "norm": {"eps": 1e-5},
           "layers": [_pair((6, 2, 64, 64, 0.12, _rot(10000.0, 64, (16.0, 256, 32.0, 1.0))), (4, 4, 32, 64, 4), _moe(8, 2, 64), (0.6, 1.1)),
                      _mem(4, 32, 64, 15.0, _moe(8, 3, 128)),
                      _pair((3, 3, 128, 128, 0.09, _rot(500000.0, 64)), (6, 2, 64, 32, 5), None, (0.8, 0.8))]},
    # the same kernels with every expert chosen, so that bfloat16 runs compare at every position; heads padded up to 64 and 128
    "nf": {"architecture": "Nipizen", "vocab": 256, "width": 128, "norm": {"eps": 1e-5},
           "layers": [_pair((4, 2, 48, 64, 0.15, _rot(3000.0, 32, (2.0, 128, 4.0, 2.0))), (2, 1, 128, 64, 4), _moe(3, 3, 256), (0.9, 0.6)),
                      _pair((2, 2, 96, 40, 0.1, _rot(10000.0, 96, (8.0, 100, 1.0, 1.0))), (4, 4, 40, 20, 2), _moe(1, 1, 64), (0.4, 1.0)),
                      _mem(1, 64, 128, 8.0)]},
    # the least there can be
    "nd": {"architecture": "Nipizen", "vocab": 50, "width": 32, "norm": {"eps": 1e-5},
           "layers": [_pair((1, 1, 4, 6, 0.4, _rot(20.0, 2)), (1, 1, 4, 4, 2))]},
    # sizes no vectorised kernel takes, five heads on one
    "ne": {"architecture": "Nipizen", "vocab": 71, "width": 38, "norm": {"eps": 1e-4},
           "layers": [_pair((5, 1, 10, 7, 0.3, _rot(30.0, 6, (3.0, 20, 2.0, 0.3))), (2, 2, 7, 5, 4), _moe(5, 3, 10), (1.0, 0.7)),
                      _mem(2, 6, 5, 1.0, _moe(3, 2, 13)),
                      _pair((2, 2, 6, 9, 0.5, _rot(40.0, 4)), (6, 2, 5, 3, 3), _moe(2, 1, 10), (0.6, 0.6))]},
}

RANKS = {"na": (6, 9), "nb": (16, 8), "nc": (32, 24), "nf": (40, 20), "nd": (1, 1), "ne": (7, 4)}      # rows of a1 and of g1


def bf16_round(a: np.ndarray) -> np.ndarray:
    return torch.from_numpy(np.asarray(a, dtype=np.float32)).to(torch.bfloat16).float().numpy()


def make_weights(cfg: dict, seed: int, ranks=(8, 8)) -> dict[str, np.ndarray]:
    """Seeded weights that bfloat16 holds exactly, as float32, by tensor name."""
    import zinfer_b200 as z
    from zinfer_b200.config.registry import build_model

    rng = np.random.default_rng(seed)
    model = build_model(z.config_from_dict(cfg))
    W = {}
    for name, spec in model.weight_specs().items():
        rank = ranks[0] if ".a1" in name or ".a2" in name else ranks[1]
        shape = tuple(rank if s < 0 else s for s in spec.shape)
        if name.endswith(".A_log"):
            W[name] = bf16_round(rng.uniform(-4.0, 0.0, shape))
        elif name.endswith(".dt_bias"):
            W[name] = bf16_round(rng.normal(-1.0, 1.0, shape))
        elif name.endswith(".f.b"):
            W[name] = bf16_round(rng.normal(3.0, 1.5, shape))
        elif name.endswith(".i.b"):
            W[name] = bf16_round(rng.normal(-1.0, 1.5, shape))
        elif name.endswith(".b") and len(shape) == 1:
            W[name] = bf16_round(rng.normal(0, 0.2, shape))
        elif "norm" in name:
            W[name] = bf16_round(1.0 + rng.normal(0, 0.2, shape))
        elif name.endswith(".conv"):
            W[name] = bf16_round(rng.normal(0, 1.0, shape) * shape[1] ** -0.5 + np.eye(1, shape[1], shape[1] - 1)[0])
        elif name == "embed":
            W[name] = bf16_round(rng.normal(0, 1.0, shape))
        elif name.endswith((".router", ".mix.i", ".mix.f")):
            W[name] = bf16_round(rng.normal(0, (3.0 if name.endswith(".router") else 1.5) * shape[-1] ** -0.5, shape))
        else:
            W[name] = bf16_round(rng.normal(0, shape[-1] ** -0.5, shape))
    return W


def write_folder(folder, cfg: dict, W: dict[str, np.ndarray]) -> Path:
    from zinfer_b200.weights import write_safetensors

    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    write_safetensors(folder / "model.safetensors", {n: torch.from_numpy(a).to(torch.bfloat16) for n, a in W.items()})
    return folder


CLOSE_CALL = 0.02       # a router choice whose margin (in score) is below this may fall either way in bfloat16


def plain_logits(cfg: dict, W: dict[str, np.ndarray], tokens):
    """(logits [n, vocab], safe): the plain implementation's logits and the number of leading positions before the first token
    whose expert choice is a close call.  In bfloat16 such a token may take another expert, and it and every later position then
    differ by far more than rounding; positions before it cannot be affected."""
    margins = [np.inf] * len(tokens)
    logits = P.forward(cfg, {n: a.astype(np.float64) for n, a in W.items()}, list(tokens), margins=margins)
    close = [t for t, m in enumerate(margins) if m < CLOSE_CALL]
    return logits, (close[0] if close else len(tokens))


def tokens_for(cfg: dict, seed: int, n: int) -> list[int]:
    return np.random.default_rng(seed).integers(0, cfg["vocab"], size=n).tolist()


TOL = {"float32": 5e-5, "bfloat16": 4e-2}


def rel_err(got, ref) -> float:
    got, ref = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    scale = float(np.abs(ref).max())
    assert scale > 0 and got.shape == ref.shape, (got.shape, ref.shape)
    return float(np.abs(got - ref).max()) / scale
