"""Mamba-2 mixer: a linear recurrence over a matrix state per head whose decay and input share follow from one learned step
size per head and token (state-space duality; Dao and Gu, "Transformers are SSMs").

Per head h of H (N state channels, e value channels, group g(h) = floor(h / (H / G)) of G), from one projection of the input
into [z (H*e) | x (H*e) | B (G*N) | C (G*N) | dt (H)]:

    x, B, C  <- silu(causal convolution per channel (K taps, bias))
    dt_t     <- softplus(dt_t + dt_bias_h)
    S_t      =  exp(-exp(A_log_h) dt_t) S_{t-1} + dt_t B_t x_t^T            y_t = S_t^T C_t + D_h x_t

The heads' y, concatenated, are multiplied by silu(z), normalised by the root mean square of each of `norm_groups` equal
parts, multiplied by a weight and projected.

The projection leaves its contraction as float32; convolution, step sizes, decays, state, sums, gate and norm are float32 in
both run dtypes.  The call's per-sequence state holds the convolution's last K-1 inputs followed by S.  Prompt steps and
single-token steps run the same kernels, from the state the step before left: `kernels.seqconv`, `kernels.ssd_scan` (the
stepped form of the recurrence kernel that also serves `Hgrn2` and `Retention`) and `kernels.gated_group_norm`."""
from __future__ import annotations

import torch

from .. import kernels
from .base import MIXERS, Mixer, StateRequest, WeightSpec
from .linear import linear, pad_rows


class Mamba2(Mixer):
    capture_safe = True
    takes_pending_norm = True
    sums_through_linear = True

    def __init__(self, hidden: int, n_heads: int, value_dim: int, state_dim: int, groups: int, taps: int, norm_groups: int,
                 in_name: str, conv_name: str, conv_bias_name: str, dt_bias_name: str, a_log_name: str, skip_name: str,
                 norm_name: str, out_name: str, norm_eps: float = 1e-5):
        if n_heads % groups:
            raise ValueError(f"mamba2: {n_heads} heads are not a multiple of {groups} groups")
        if (n_heads * value_dim) % norm_groups:
            raise ValueError(f"mamba2: {n_heads * value_dim} values cannot be normalised in {norm_groups} equal parts")
        if taps < 1:
            raise ValueError(f"mamba2: a convolution needs at least one tap, got {taps}")
        self.hidden, self.n_heads, self.value_dim, self.state_dim, self.groups = hidden, n_heads, value_dim, state_dim, groups
        self.taps, self.norm_groups, self.eps = int(taps), int(norm_groups), float(norm_eps)
        self.in_name, self.conv_name, self.conv_bias_name = in_name, conv_name, conv_bias_name
        self.dt_bias_name, self.a_log_name, self.skip_name = dt_bias_name, a_log_name, skip_name
        self.norm_name, self.out_name = norm_name, out_name
        self.w_in = self.w_out = self.conv = self.conv_bias = self.dt_bias = self.a_log = self.skip = self.norm = None

    @property
    def inner(self):
        return self.n_heads * self.value_dim

    @property
    def channels(self):
        return self.inner + 2 * self.groups * self.state_dim

    @property
    def conv_state(self):
        return (self.taps - 1) * self.channels

    def weight_specs(self):
        H = self.n_heads
        return [WeightSpec(self.in_name, (self.inner + self.channels + H, self.hidden)),
                WeightSpec(self.conv_name, (self.channels, self.taps), role="vector"),
                WeightSpec(self.conv_bias_name, (self.channels,), role="vector"),
                WeightSpec(self.dt_bias_name, (H,), role="vector"),
                WeightSpec(self.a_log_name, (H,), role="vector"),
                WeightSpec(self.skip_name, (H,), role="vector", init="norm"),
                WeightSpec(self.norm_name, (self.inner,), role="vector", init="norm"),
                WeightSpec(self.out_name, (self.hidden, self.inner))]

    def load(self, weights, dtype, device):
        self.w_in, self.w_out = pad_rows(weights[self.in_name]), weights[self.out_name]
        self.conv = weights[self.conv_name].t().contiguous()            # [taps, channels]: a tap's channels side by side
        self.conv_bias, self.norm = weights[self.conv_bias_name], weights[self.norm_name]
        self.dt_bias, self.a_log, self.skip = (weights[n] for n in (self.dt_bias_name, self.a_log_name, self.skip_name))

    def state_request(self):
        size = self.conv_state + self.n_heads * self.state_dim * self.value_dim
        return StateRequest((-(-size // 4) * 4,), torch.float32)        # whole 16-byte pieces per slot

    def check(self, dtype, page_size):
        if self.state_dim > kernels.hgrn2_max_dim():
            raise ValueError(f"mamba2: {self.state_dim} state channels exceed the supported {kernels.hgrn2_max_dim()}")
        if self.taps > kernels.seqconv_max_taps():
            raise ValueError(f"mamba2: {self.taps} taps exceed the supported {kernels.seqconv_max_taps()}")

    def forward(self, ctx, call, xn, out, accumulate):
        inner, ch, H = self.inner, self.channels, self.n_heads
        p = linear(xn, self.w_in, out_dtype=torch.float32)              # [z | x | B | C | dt (| padding)]
        conv = call.state[:, :self.conv_state].unflatten(1, (self.taps - 1, ch))
        rec = call.state[:, self.conv_state:self.conv_state + H * self.state_dim * self.value_dim]
        xbc = kernels.seqconv(p[:, inner:inner + ch], conv, self.conv, ctx.tok_seq, ctx.cu_q, ctx.seq_slot, ctx.n_seqs,
                              torch.float32, residual=False, single_token=ctx.is_decode, bias=self.conv_bias, silu=True)
        y = kernels.ssd_scan(xbc, p[:, inner + ch:inner + ch + H], self.dt_bias, self.a_log, self.skip, rec, ctx.cu_q, ctx.seq_slot,
                             ctx.n_seqs, H, self.groups, self.state_dim, self.value_dim)
        g = kernels.gated_group_norm(y, p[:, :inner], self.norm, self.norm_groups, self.eps, ctx.dtype)
        linear(g, self.w_out, out=out, accumulate=accumulate)


MIXERS.register("mamba2", Mamba2)
