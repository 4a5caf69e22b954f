"""Token embedding and output head.  x_t = E[token_t] (times a scale, 1 here:
src/model.zig:2352-2358, 466); logits = xn W_out^T in float32 with W_out the head tensor or
the embedding itself when tied (src/model.zig:595-598, 2490).

Options other designs use: a learned position table whose row for the token's position is
added to the embedding (unscaled, float32), a table of rows for pairs (token before, token), a soft cap on the logits,
logits <- cap * tanh(logits / cap), and a constant the logits are multiplied by (`scale`, applied last).

Pair rows (`bigram` = (name, buckets, mul_prev, mul_cur)): row (token before * mul_prev + token * mul_cur) mod buckets of a
table of buckets + 1 rows is added, unscaled; the last row for a sequence's first token.  The token before is per-sequence
state of the embedding (`state_request`), so that a sequence cut into steps embeds as if it were whole.
`copies`: the rows go to so many planes [copies, tokens, width], the residual streams of a model that keeps streams."""
from __future__ import annotations

import torch

from .. import kernels
from .base import Part, StateRequest, WeightSpec
from .linear import linear


class TokenEmbedding(Part):
    def __init__(self, vocab: int, dim: int, weight_name: str, scale: float = 1.0,
                 position_name: str | None = None, max_positions: int = 0, bigram: tuple[str, int, int, int] | None = None,
                 copies: int | None = None):
        """position_name: a learned table [max_positions, dim] whose row of the token's position is added."""
        self.vocab, self.dim, self.weight_name, self.scale = vocab, dim, weight_name, float(scale)
        self.position_name, self.max_positions = position_name, int(max_positions)
        if position_name is not None and self.max_positions <= 0:
            raise ValueError("a position table needs its number of positions")
        if bigram is not None and int(bigram[1]) < 1:
            raise ValueError(f"pair rows: {bigram[1]} buckets")
        self.bigram, self.copies = bigram, copies
        self.weight = self.positions = self.pairs = None

    def weight_specs(self):
        specs = [WeightSpec(self.weight_name, (self.vocab, self.dim))]
        if self.position_name is not None:
            specs.append(WeightSpec(self.position_name, (self.max_positions, self.dim)))
        if self.bigram is not None:
            specs.append(WeightSpec(self.bigram[0], (int(self.bigram[1]) + 1, self.dim)))
        return specs

    def state_request(self):
        """Fixed per-sequence state the embedding needs (the last token of the sequence), or None."""
        return StateRequest((1,), torch.int32) if self.bigram is not None else None

    def load(self, weights, dtype, device):
        self.weight = weights[self.weight_name]
        self.positions = weights[self.position_name] if self.position_name is not None else None
        self.pairs = weights[self.bigram[0]] if self.bigram is not None else None

    def forward(self, ctx, tokens: torch.Tensor, out: torch.Tensor | None = None,
                state: torch.Tensor | None = None) -> torch.Tensor:
        pairs = batch = None
        if self.pairs is not None:
            pairs = (self.pairs, self.bigram[2], self.bigram[3])
            batch = (ctx.tok_seq, ctx.tok_pos, ctx.cu_q, ctx.seq_slot, ctx.n_seqs)
        return kernels.embed(tokens, self.weight, ctx.status, self.scale, self.positions,
                             ctx.tok_pos if self.positions is not None else None, out=out, bigram=pairs, batch=batch, prev=state,
                             single_token=ctx.is_decode, copies=self.copies)


class LMHead(Part):
    """`weight_name` None ties the head to `embedding`."""

    def __init__(self, vocab: int, dim: int, weight_name: str | None, embedding: TokenEmbedding | None = None,
                 softcap: float | None = None, scale: float = 1.0):
        if weight_name is None and embedding is None:
            raise ValueError("a tied head needs the embedding it is tied to")
        if softcap is not None and not softcap > 0:
            raise ValueError(f"a logit cap must be positive, got {softcap}")
        self.vocab, self.dim, self.weight_name, self.embedding = vocab, dim, weight_name, embedding
        self.softcap = None if softcap is None else float(softcap)
        self.scale = float(scale)
        self.weight = None

    def weight_specs(self):
        return [] if self.weight_name is None else [WeightSpec(self.weight_name, (self.vocab, self.dim))]

    def load(self, weights, dtype, device):
        self.weight = None if self.weight_name is None else weights[self.weight_name]

    takes_pending_norm = True

    def forward(self, ctx, xn, out: torch.Tensor | None = None) -> torch.Tensor:
        """float32 logits of the rows of xn (a tensor, or a norm still pending), into `out` if given."""
        w = self.weight if self.weight is not None else self.embedding.weight
        logits = linear(xn, w, out=out, out_dtype=torch.float32)
        if self.softcap is not None:
            kernels.softcap(logits, self.softcap)
        if self.scale != 1.0:
            kernels.scale_(logits, self.scale)
        return logits
