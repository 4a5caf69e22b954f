"""Gated delta rule mixer: a linear recurrence over a matrix state per head that forgets per key channel and writes only what
the key does not yet read (delta networks with a gate; Yang, Kautz and Hatamizadeh, "Gated Delta Networks: Improving Mamba2
with Delta Rule").

Per head h of H (d key channels, e value channels, queries and keys of head floor(h / (H / G)) of G), from the input x_t:

    q, k, v   <- silu(causal convolution per channel (K taps, no bias)) of W_q x, W_k x, W_v x
    q, k      <- q / sqrt(sum q^2 + 1e-6) * d^-1/2,  k / sqrt(sum k^2 + 1e-6)
    beta_t    =  sigmoid(W_b x)                                           one per head
    g_t       =  exp(-exp(A_log_h) softplus(W_a2 W_a1 x + dt_bias))       one per head and key channel
    S <- diag(g_t) S      u = beta_t (v - S^T k)      S <- S + k u^T      o_t = S^T q

Each head's o_t is divided by its root mean square, multiplied by one weight vector [e] shared by the heads and by
sigmoid(W_g2 W_g1 x); the concatenated heads are projected by W_o.  The two inner widths (rows of W_a1 and W_g1) are the
tensors' own.

q, k, v, both inner widths of the low-rank maps and beta's logits are one contraction with a float32 result; one block-diagonal
contraction (float32 result) leads out of both inner widths.  Convolution, unit vectors, decays, beta, state, sums,
norm and gate are float32 in both run dtypes (`kernels.seqconv`, `kernels.delta_scan`, `kernels.unit_norm_gate`).  The call's
per-sequence state holds the convolution's last K - 1 inputs followed by the matrices.  Prompt steps and single-token steps run
the same recurrence kernel from the state the step before left."""
from __future__ import annotations

import torch

from .. import kernels
from .base import ANY_SIZE, MIXERS, Mixer, StateRequest, WeightSpec
from .linear import linear, pad_rows

LOW_RANK_ALIGN = 8       # the inner widths together, brought up to what the tensor-core contractions take with zeros


class GatedDelta(Mixer):
    capture_safe = True
    takes_pending_norm = True
    sums_through_linear = True

    def __init__(self, hidden: int, n_heads: int, n_kv_heads: int, dim: int, value_dim: int, taps: int, q_name: str, k_name: str,
                 v_name: str, q_conv_name: str, k_conv_name: str, v_conv_name: str, beta_name: str, a_log_name: str, a1_name: str,
                 a2_name: str, dt_bias_name: str, g1_name: str, g2_name: str, norm_name: str, out_name: str,
                 norm_eps: float = 1e-5):
        if n_heads % n_kv_heads:
            raise ValueError(f"gated delta rule: {n_heads} heads are not a multiple of {n_kv_heads} query/key heads")
        if taps < 1:
            raise ValueError(f"gated delta rule: a convolution needs at least one tap, got {taps}")
        self.hidden, self.n_heads, self.n_kv, self.dim, self.value_dim = hidden, n_heads, n_kv_heads, dim, value_dim
        self.taps, self.eps = int(taps), float(norm_eps)
        self.proj_names, self.conv_names = (q_name, k_name, v_name, beta_name), (q_conv_name, k_conv_name, v_conv_name)
        self.a_log_name, self.dt_bias_name = a_log_name, dt_bias_name
        self.a1_name, self.a2_name, self.g1_name, self.g2_name = a1_name, a2_name, g1_name, g2_name
        self.norm_name, self.out_name = norm_name, out_name
        self.w_in = self.w_high = self.w_out = self.conv = self.a_log = self.dt_bias = self.norm = None

    @property
    def key_dim(self):
        return self.n_kv * self.dim

    @property
    def decay_dim(self):
        return self.n_heads * self.dim

    @property
    def out_dim(self):
        return self.n_heads * self.value_dim

    @property
    def channels(self):
        return 2 * self.key_dim + self.out_dim

    @property
    def conv_floats(self):
        """Floats of the convolution's state, brought up so that the matrices behind it start on 16 bytes."""
        return -(-(self.taps - 1) * self.channels // 4) * 4

    def weight_specs(self):
        D, kd, od = self.hidden, self.key_dim, self.out_dim
        q, k, v, b = self.proj_names
        specs = [WeightSpec(q, (kd, D)), WeightSpec(k, (kd, D)), WeightSpec(v, (od, D)), WeightSpec(b, (self.n_heads, D))]
        specs += [WeightSpec(n, (w, self.taps), role="vector") for n, w in zip(self.conv_names, (kd, kd, od))]
        specs += [WeightSpec(self.a_log_name, (self.n_heads,), role="vector"),
                  WeightSpec(self.a1_name, (ANY_SIZE, D), free_size=self.dim),
                  WeightSpec(self.a2_name, (self.decay_dim, ANY_SIZE), free_size=self.dim),
                  WeightSpec(self.dt_bias_name, (self.decay_dim,), role="vector"),
                  WeightSpec(self.g1_name, (ANY_SIZE, D), free_size=self.value_dim),
                  WeightSpec(self.g2_name, (od, ANY_SIZE), free_size=self.value_dim),
                  WeightSpec(self.norm_name, (self.value_dim,), role="vector", init="norm"),
                  WeightSpec(self.out_name, (D, od))]
        return specs

    def load(self, weights, dtype, device):
        a1, a2, g1, g2 = (weights[n] for n in (self.a1_name, self.a2_name, self.g1_name, self.g2_name))
        for inner, outer, name in ((a1, a2, self.a1_name), (g1, g2, self.g1_name)):
            if inner.shape[0] != outer.shape[1]:
                raise ValueError(f"tensor '{name}' has {inner.shape[0]} rows, the matrix behind it {outer.shape[1]} columns")
        ra, rg = a1.shape[0], g1.shape[0]
        r = -(-(ra + rg) // LOW_RANK_ALIGN) * LOW_RANK_ALIGN
        q, k, v, beta = (weights[n] for n in self.proj_names)
        self.rank = r
        self.w_in = pad_rows(torch.cat([q, k, v, a1, g1, a1.new_zeros((r - ra - rg, self.hidden)), beta], dim=0).contiguous())
        self.w_high = a2.new_zeros((self.decay_dim + self.out_dim, r))
        self.w_high[:self.decay_dim, :ra] = a2
        self.w_high[self.decay_dim:, ra:ra + rg] = g2
        self.w_high = pad_rows(self.w_high)
        self.conv = torch.cat([weights[n] for n in self.conv_names], dim=0).t().contiguous()   # [taps, channels]
        self.a_log, self.dt_bias, self.norm = (weights[n] for n in (self.a_log_name, self.dt_bias_name, self.norm_name))
        self.w_out = weights[self.out_name]

    def state_request(self):
        size = self.conv_floats + kernels.delta_state_floats(self.n_heads, self.dim, self.value_dim)
        return StateRequest((-(-size // 4) * 4,), torch.float32)        # whole 16-byte pieces per slot

    def check(self, dtype, page_size):
        if self.dim > kernels.delta_max_dim():
            raise ValueError(f"gated delta rule: {self.dim} key channels exceed the supported {kernels.delta_max_dim()}")
        if self.taps > kernels.seqconv_max_taps():
            raise ValueError(f"gated delta rule: {self.taps} taps exceed the supported {kernels.seqconv_max_taps()}")

    def forward(self, ctx, call, xn, out, accumulate):
        H, G, d, e, ch = self.n_heads, self.n_kv, self.dim, self.value_dim, self.channels
        r = self.rank
        p = linear(xn, self.w_in, out_dtype=torch.float32)                   # [q | k | v | inner widths | beta (| padding)]
        ag = linear(kernels.cast_rows(p[:, ch:ch + r], ctx.dtype), self.w_high, out_dtype=torch.float32)   # [decays | gate (| padding)]
        conv = call.state[:, :(self.taps - 1) * ch].unflatten(1, (self.taps - 1, ch))
        rec = call.state[:, self.conv_floats:self.conv_floats + kernels.delta_state_floats(H, d, e)]
        qkv = kernels.seqconv(p[:, :ch], conv, self.conv, ctx.tok_seq, ctx.cu_q, ctx.seq_slot, ctx.n_seqs, torch.float32,
                              residual=False, single_token=ctx.is_decode, silu=True)
        o = kernels.delta_scan(qkv, ag, p[:, ch + r:ch + r + H], self.a_log, self.dt_bias, rec, ctx.tok_seq, ctx.cu_q, ctx.seq_slot, ctx.n_seqs, H, G, d, e,
                               single_token=ctx.is_decode)
        on = kernels.unit_norm_gate(o, ag[:, self.decay_dim:], H, self.eps, ctx.dtype, weight=self.norm, sigmoid=True)
        linear(on, self.w_out, out=out, accumulate=accumulate)


MIXERS.register("gated_delta", GatedDelta)
