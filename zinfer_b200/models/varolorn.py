"""Varolorn: a pre-norm decoder on several residual streams (hyper-connections) that mixes two kinds of layers in any order:
the Mamba-2 recurrence, and grouped-query softmax attention without a rotation, whose queries see only their own stretch of
positions and whose scores are moved by a learned number per (distance bucket, head), with biases in its projections, normed
query and key heads, values mixed with those of the first attention layer, and a gate per head.  A dense gated
feed-forward (relu) follows a mixer or not.  Norm weights are stored around zero; a row for the pair (token before, token) is
added to the scaled token row; the head is the embedding table.

Per layer i the tensors are `l<i>.*`.  Every part is a general part of `parts/`; this file only names tensors and
passes the configuration's numbers on."""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.varolorn import VarolornConfig
from ..parts import (GqaAttention, LMHead, Mamba2, PreNormBlock, ReluGLU, RMSNorm, StreamBlock, StreamNorm, TokenEmbedding)
from .model import Model


def build_varolorn(cfg: VarolornConfig) -> Model:
    D, eps, S = cfg.hidden_size, cfg.norm_eps, cfg.streams
    b = cfg.bigram
    embedding = TokenEmbedding(cfg.vocab_size, D, "embed", scale=cfg.embedding_scale, copies=S or None,
                               bigram=None if b is None else ("bigram", b.buckets, b.mul_prev, b.mul_cur))
    first_values = cfg.first_value_layer()
    layers = []
    for i, L in enumerate(cfg.layers):
        p, m = f"l{i}.", L.mixer
        a = p + "mix."
        if L.type == "mamba2":
            mixer = Mamba2(D, m.heads, m.vdim, m.state, m.groups, m.conv, m.norm_groups, a + "in", a + "conv", a + "conv.b",
                           a + "dt_bias", a + "A_log", a + "D", a + "norm", a + "o", norm_eps=eps)
        else:
            mixer = GqaAttention(D, m.heads, m.kv_heads, m.dim, a + "q", a + "k", a + "v", a + "o", q_norm_name=a + "q.norm",
                                 k_norm_name=a + "k.norm", norm_eps=eps, scale=m.scale, value_dim=m.vdim, pad_heads=True,
                                 bias_names=(a + "q.b", a + "k.b", a + "v.b", a + "o.b"), distance_rows=(a + "rel", m.bias_max),
                                 chunk=m.chunk, head_gate_name=a + "g",
                                 value_mix=(a + "vmix", i == first_values) if m.v_mix else None)
        ffn = None if L.ff is None else ReluGLU(D, L.ff, p + "mlp.gate", p + "mlp.up", p + "mlp.down")
        if S:
            def norm(q):
                return StreamNorm(D, eps, f"{p}norm{q}", S, read_name=f"{p}hc{q}.in", one_plus=True)

            def write(q):
                return (f"{p}hc{q}.mix", f"{p}hc{q}.out")

            layers.append(StreamBlock(norm(1), mixer, write(1), *((norm(2), ffn, write(2)) if ffn is not None else ())))
        else:
            layers.append(PreNormBlock(RMSNorm(D, eps, p + "norm1", one_plus=True), mixer,
                                       RMSNorm(D, eps, p + "norm2", one_plus=True) if ffn is not None else None, ffn))
    final = StreamNorm(D, eps, "final.norm", S, one_plus=True) if S else RMSNorm(D, eps, "final.norm", one_plus=True)
    return Model(cfg, embedding, layers, final, LMHead(cfg.vocab_size, D, None, embedding))


register_architecture("Varolorn", VarolornConfig, build_varolorn)
