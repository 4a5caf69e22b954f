"""Nipizen: a pre-norm decoder (layer norms with a weight and no bias) that mixes two kinds of layers in any order.  A pair of
mixers side by side, summed with a fixed factor each: grouped-query softmax attention (biases on q, k and v, norms over the whole
q and k projections, a rotation with YaRN frequencies, a sigmoid gate on every output value) and the gated delta rule (short
convolutions, unit queries and keys, a decay per head and key channel).  Or an mLSTM, a matrix memory with exponential gates.
The feed-forward, if a layer has one, is a mixture of ungated experts (squared relu) picked by sigmoid scores that are not
renormalised and multiply what an expert reads.  The head is the embedding table.

Per layer i the tensors are `l<i>.*`.  Every part is a general part of `parts/`; this file only names tensors and passes the
configuration's numbers on."""
from __future__ import annotations

from ..config.nipizen import NipizenConfig
from ..config.registry import register_architecture
from ..parts import (GatedDelta, GqaAttention, LayerNorm, LMHead, MixerPair, MLstm, PreNormBlock, RotaryEncoding, RoutedMoE,
                     TokenEmbedding)
from .model import Model


def build_nipizen(cfg: NipizenConfig) -> Model:
    D, eps = cfg.hidden_size, cfg.norm_eps
    embedding = TokenEmbedding(cfg.vocab_size, D, "embed")
    layers = []
    for i, L in enumerate(cfg.layers):
        p = f"l{i}."
        a = p + "mix."
        if L.type == "mlstm":
            m = L.mlstm
            mixer = MLstm(D, m.heads, m.dim, m.vdim, m.gate_cap, a + "q", a + "k", a + "v", a + "i", a + "i.b", a + "f", a + "f.b",
                          a + "g", a + "norm", a + "o", norm_eps=eps)
        else:
            l, r, s, t = L.left, L.right, a + "left.", a + "right."
            position = RotaryEncoding(l.dim, l.rot_base, n_rot=l.rot_dims, yarn=l.yarn) if l.rot_dims else None
            left = GqaAttention(D, l.heads, l.kv_heads, l.dim, s + "q", s + "k", s + "v", s + "o", q_norm_name=s + "q.norm",
                                k_norm_name=s + "k.norm", norm_eps=eps, position=position, scale=l.scale, value_dim=l.vdim,
                                qk_norm_span="all", bias_names=(s + "q.b", s + "k.b", s + "v.b", None), value_gate_name=s + "g",
                                pad_heads=True)
            right = GatedDelta(D, r.heads, r.kv_heads, r.dim, r.vdim, r.conv, t + "q", t + "k", t + "v", t + "q.conv", t + "k.conv",
                               t + "v.conv", t + "b", t + "A_log", t + "a1", t + "a2", t + "dt_bias", t + "g1", t + "g2", t + "norm",
                               t + "o", norm_eps=eps)
            mixer = MixerPair(D, left, right, scales=(L.left_scale, L.right_scale))
        ffn = None
        if L.mlp is not None:
            f = p + "mlp."
            ffn = RoutedMoE(D, L.mlp.ff, L.mlp.experts, L.mlp.top, f + "router", lambda e, f=f: (f"{f}e{e}.up", f"{f}e{e}.down"),
                            score="sigmoid", renormalize=False, weight_input=True, act="relu_squared")
        layers.append(PreNormBlock(LayerNorm(D, eps, p + "norm1"), mixer, LayerNorm(D, eps, p + "norm2") if ffn is not None else None,
                                   ffn))
    return Model(cfg, embedding, layers, LayerNorm(D, eps, "final.norm"), LMHead(cfg.vocab_size, D, None, embedding),
                 ignorable_weights=[f"l{i}.norm2" for i, L in enumerate(cfg.layers) if L.mlp is None])


register_architecture("Nipizen", NipizenConfig, build_nipizen)
