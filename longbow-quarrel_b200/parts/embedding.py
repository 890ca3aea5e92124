"""Token embedding and output head.

Embedding: row `token` of the table, no multiplier unless asked for, promoted to the 32-bit residual
stream (internal/device/kernels.metal:465-467; internal/engine/engine.go:1365-1375).
Head: logits = n . W^T in 32-bit (internal/engine/engine.go:1561;
internal/device/kernels.metal:1172-1194), reading the embedding table when the
model ties them (internal/engine/engine.go:1108-1111).
"""
from __future__ import annotations

import torch

from ..kernels import linear, ops
from ..weights.spec import WeightSpec
from .base import Part, Runtime, StateNeed
from .registry import make_part, register_part
from .spec import PartSpec


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    graph_safe = True

    def __init__(self, runtime: Runtime, vocab_size: int, hidden_size: int, name: str, norm: PartSpec | None = None, scale: float = 1.0):
        """norm: an RMS norm with a gain that the rows pass before they become the stream.  scale: the rows are multiplied by
        this constant, in 32-bit (without a norm)."""
        self.scale = float(scale)
        if norm is not None and self.scale != 1.0:
            raise ValueError("token_embedding: a multiplier on the rows or a norm, not both")
        self.runtime, self.vocab_size, self.hidden_size, self.name = runtime, vocab_size, hidden_size, name
        self.norm = make_part("norm", norm, runtime) if norm is not None else None
        if self.norm is not None and not (hasattr(self.norm, "gain") and hasattr(self.norm, "eps") and not hasattr(self.norm, "bias")):
            raise ValueError("token_embedding: the rows' norm must be an RMS norm with a gain")
        self.emits_stream = self.norm is not None      # forward(emit_stream=True) also returns the rows in the activations' dtype
        self.kernel_libraries = ("post_norm",) if self.norm is not None else ()
        self.table: torch.Tensor | None = None

    def weights(self):
        out = {self.name: WeightSpec((self.vocab_size, self.hidden_size))}
        if self.norm is not None:
            out.update(self.norm.weights())
        return out

    def load(self, tensors):
        self.table = tensors[self.name]
        if self.norm is not None:
            self.norm.load({n: tensors[n] for n in self.norm.weights()})

    def forward(self, tokens: torch.Tensor, emit_stream: bool = False):
        if self.norm is None:
            return ops.embedding(self.table, tokens, scale=self.scale)
        x, rows = ops.embedding_norm(self.table, tokens, self.norm.gain, self.norm.eps, self.runtime.act_dtype if emit_stream else None)
        return (x, rows) if emit_stream else x


@register_part("embedding", "pair_hash_embedding")
class PairHashEmbedding(Part):
    """Token embedding plus a row of a second table chosen by the pair (token before, token):

        x_t = table[tok_t] + pairs[(tok_(t-1) * mul_prev + tok_t * mul_cur) mod buckets]

    and `pairs[buckets]`, the table's last row, for the first token of a sequence.  The token before a step's first
    row is part of the sequence's state: one int32 per slot (`state_need`), which the step's last token replaces."""

    graph_safe = True

    def __init__(self, runtime: Runtime, vocab_size: int, hidden_size: int, name: str, pairs_name: str, buckets: int,
                 mul_prev: int, mul_cur: int):
        if buckets < 1:
            raise ValueError(f"pair_hash_embedding: {buckets} buckets")
        self.runtime, self.vocab_size, self.hidden_size = runtime, vocab_size, hidden_size
        self.name, self.pairs_name = name, pairs_name
        self.buckets, self.mul_prev, self.mul_cur = int(buckets), int(mul_prev), int(mul_cur)
        self.table: torch.Tensor | None = None
        self.pairs: torch.Tensor | None = None

    def weights(self):
        return {self.name: WeightSpec((self.vocab_size, self.hidden_size)),
                self.pairs_name: WeightSpec((self.buckets + 1, self.hidden_size))}

    def load(self, tensors):
        self.table, self.pairs = tensors[self.name], tensors[self.pairs_name]
        if self.pairs.dtype != self.table.dtype:
            self.table, self.pairs = self.table.to(torch.float32), self.pairs.to(torch.float32)

    def state_need(self):
        """The sequence's last token, kept between steps."""
        return StateNeed((), torch.int32)

    def forward(self, tokens: torch.Tensor, ctx=None, state=None) -> torch.Tensor:
        return ops.embedding_pairs(self.table, self.pairs, self.buckets, self.mul_prev, self.mul_cur, tokens, ctx.tok_pos,
                                   ctx.tok_seq, ctx.slots, ctx.cu_rows, state, ctx.B)


@register_part("head", "linear_head")
class LinearHead(Part):
    """`tied_to` names the tensor (of another part) that the head reads when it has
    none of its own; with `tied` true it never has its own."""

    graph_safe = True

    def __init__(self, runtime: Runtime, vocab_size: int, hidden_size: int, name: str, tied_to: str | None = None,
                 tied: bool = False, softcap: float | None = None):
        """softcap c: logits <- c tanh(logits / c)."""
        self.softcap = float(softcap) if softcap else None
        self.runtime, self.vocab_size, self.hidden_size = runtime, vocab_size, hidden_size
        self.name, self.tied_to, self.tied = name, tied_to, tied
        self.weight: linear.LinearWeight | None = None

    def weights(self):
        if self.tied:
            return {}
        return {self.name: WeightSpec((self.vocab_size, self.hidden_size), fallback=self.tied_to)}

    def borrows(self):
        return [self.tied_to] if self.tied_to is not None else []

    def load(self, tensors):
        w = tensors.get(self.name)
        if w is None:
            w = tensors[self.tied_to]
        self.weight = linear.LinearWeight(w)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        logits = linear.linear(h, self.weight, torch.float32)
        return ops.softcap(logits, self.softcap) if self.softcap else logits
