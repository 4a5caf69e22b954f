"""mLSTM mixer: a matrix memory with exponential gates and a normaliser (Beck et al., "xLSTM: Extended Long Short-Term Memory").

Per head (H heads, d query/key channels, e value channels), from the input x_t:

    q = W_q x * d^-1/2      k = W_k x      v = W_v x
    i = c tanh((W_i x + b_i) / c)      f = log sigmoid(c tanh((W_f x + b_f) / c))      logarithms of the gates, c the cap
    m_t = max(f + m_{t-1}, i), m_0 = 0
    S_t = exp(f + m_{t-1} - m_t) S_{t-1} + exp(i - m_t) k v^T      n_t likewise with k alone
    o_t = S_t^T q / (max(|n_t . q|, exp(-m_t)) + 1e-6)

Each head's o_t is divided by its root mean square; the concatenated heads are multiplied by one weight and by
sigmoid(W_g x) and projected by W_o.

All projections but the last are one contraction with a float32 result; gates, maxima, state, sums, the quotient, norm and
output gate are float32 in both run dtypes (`kernels.mlstm_scan`, the capped form of the recurrence kernel that also serves
`Hgrn2`, `Retention` and `Mamba2`; `kernels.unit_norm_gate`).  The normaliser is one more value column, of ones.  The call's
per-sequence state holds the matrices and the running maxima; prompt steps and single-token steps run the same kernels."""
from __future__ import annotations

import torch

from .. import kernels
from .base import MIXERS, Mixer, StateRequest, WeightSpec
from .linear import linear, pad_rows


class MLstm(Mixer):
    capture_safe = True
    takes_pending_norm = True
    sums_through_linear = True

    def __init__(self, hidden: int, n_heads: int, dim: int, value_dim: int, gate_cap: float, q_name: str, k_name: str, v_name: str,
                 i_name: str, i_bias_name: str, f_name: str, f_bias_name: str, gate_name: str, norm_name: str, out_name: str,
                 norm_eps: float = 1e-5):
        if not gate_cap > 0:
            raise ValueError(f"mlstm: the cap of the gates must be positive, got {gate_cap}")
        self.hidden, self.n_heads, self.dim, self.value_dim = hidden, n_heads, dim, value_dim
        self.cap, self.eps = float(gate_cap), float(norm_eps)
        self.q_name, self.k_name, self.v_name, self.i_name, self.f_name = q_name, k_name, v_name, i_name, f_name
        self.i_bias_name, self.f_bias_name, self.gate_name = i_bias_name, f_bias_name, gate_name
        self.norm_name, self.out_name = norm_name, out_name
        self.w_in = self.w_out = self.i_bias = self.f_bias = self.norm = None

    @property
    def key_dim(self):
        return self.n_heads * self.dim

    @property
    def out_dim(self):
        return self.n_heads * self.value_dim

    def weight_specs(self):
        D, H = self.hidden, self.n_heads
        return [WeightSpec(self.q_name, (self.key_dim, D)), WeightSpec(self.k_name, (self.key_dim, D)),
                WeightSpec(self.v_name, (self.out_dim, D)), WeightSpec(self.gate_name, (self.out_dim, D)),
                WeightSpec(self.i_name, (H, D)), WeightSpec(self.f_name, (H, D)),
                WeightSpec(self.i_bias_name, (H,), role="vector"), WeightSpec(self.f_bias_name, (H,), role="vector"),
                WeightSpec(self.norm_name, (self.out_dim,), role="vector", init="norm"),
                WeightSpec(self.out_name, (D, self.out_dim))]

    def load(self, weights, dtype, device):
        names = (self.q_name, self.k_name, self.v_name, self.gate_name, self.i_name, self.f_name)
        self.w_in = pad_rows(torch.cat([weights[n] for n in names], dim=0).contiguous())
        self.w_out, self.norm = weights[self.out_name], weights[self.norm_name]
        self.i_bias, self.f_bias = weights[self.i_bias_name], weights[self.f_bias_name]

    def state_request(self):
        size = kernels.mlstm_state_floats(self.n_heads, self.dim, self.value_dim)
        return StateRequest((-(-size // 4) * 4,), torch.float32)

    def check(self, dtype, page_size):
        if self.dim > kernels.hgrn2_max_dim():
            raise ValueError(f"mlstm: {self.dim} channels per head exceed the supported {kernels.hgrn2_max_dim()}")

    def forward(self, ctx, call, xn, out, accumulate):
        H, d, e = self.n_heads, self.dim, self.value_dim
        p = linear(xn, self.w_in, out_dtype=torch.float32)              # [q | k | v | gate | i | f (| padding)]
        at = 2 * self.key_dim + 2 * self.out_dim
        state = call.state[:, :kernels.mlstm_state_floats(H, d, e)]
        o, m = kernels.mlstm_scan(p, p[:, at:at + H], p[:, at + H:at + 2 * H], self.i_bias, self.f_bias, self.cap, state, ctx.cu_q,
                                  ctx.seq_slot, ctx.n_seqs, H, d, e)
        on = kernels.unit_norm_gate(o, p[:, 2 * self.key_dim + self.out_dim:at], H, self.eps, ctx.dtype, weight=self.norm,
                                    sigmoid=True, den_log=m, out_scale=float(d) ** -0.5)
        linear(on, self.w_out, out=out, accumulate=accumulate)


MIXERS.register("mlstm", MLstm)
