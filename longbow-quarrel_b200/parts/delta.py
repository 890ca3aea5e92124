"""The gated delta rule: a mixer that keeps a matrix of fixed size per head and corrects it token by token.

Per head, with S (key size x value size, float32) carried from token to token in the cache:

    S' = diag(a_t) S_(t-1)      u_t = b_t (v_t - S'^T k_t)      S_t = S' + k_t u_t^T      o_t = S_t^T q_t

Both kinds: q, k and v each pass a short causal convolution over time per channel and silu; q and k are unit vectors per head
after it (x / sqrt(sum(x^2) + 1e-6)), q times key size^-1/2; there may be fewer q and k heads than value heads; b_t =
sigmoid(W_b h), one number per head; each head's output leaves over its root mean square, times a weight of the head's size
that all heads share, times a gate, then W_o.

"channel_delta": a_t is a vector over the head's key channels, a_t = exp(-exp(A_h) softplus(W_a2 (W_a1 h) + c)); the gate is
sigmoid(W_g2 (W_g1 h)).  "head_delta": a_t is one number per head, a_t = exp(-exp(A_h) softplus(W_a h + c_h)); the gate is
silu(W_g h).

Everything that enters the recurrence is 32-bit in both precisions: the input products hand on their 32-bit sums, and the
second product of the decays runs on the first one's sums (as two bfloat16 terms each where the tensor cores take it).
The state and the convolution's last inputs are kept per slot; steps of one token per sequence are one kernel from the
input product to the output product (`csrc/delta.cu`).
"""
from __future__ import annotations

import torch

from ..kernels import linear, ops
from ..weights.spec import WeightSpec
from .base import Mixer, Runtime, SeveralNeeds, StateNeed, StepContext
from .registry import register_part

UNIT_EPS = 1e-6        # inside the root of q's and k's unit vectors


class DeltaRule(Mixer):
    """What both kinds share: sizes, the cache entry (the state and the convolution's last inputs), the convolution's weights."""
    graph_safe = True
    returns_branch = True

    def __init__(self, runtime: Runtime, hidden_size: int, n_heads: int, key_dim: int, value_dim: int, taps: int, eps: float,
                 n_kv_heads: int | None, names: tuple, given: dict | None, most_values: int, kind: str):
        n_kv_heads = n_heads if n_kv_heads is None else n_kv_heads
        if n_heads % n_kv_heads:
            raise ValueError(f"{kind}: {n_heads} heads are not a multiple of {n_kv_heads} kv heads")
        if not 1 <= key_dim <= 256 or not 1 <= value_dim <= most_values or taps < 1:
            raise ValueError(f"{kind}: key size {key_dim} (at most 256), value size {value_dim} (at most {most_values}), {taps} taps (at least 1)")
        self.runtime, self.D, self.H, self.G, self.dk, self.dv = runtime, hidden_size, n_heads, n_kv_heads, key_dim, value_dim
        self.taps, self.eps = int(taps), float(eps)
        self.names = {n: n for n in names}
        self.names.update(given or {})
        for n in ("q", "k", "v"):
            self.names.setdefault(n + "_conv", self.names[n] + ".conv")
        self.w_in: linear.LinearWeight | None = None
        self.w_o: linear.LinearWeight | None = None
        self.taps_w = self.rate = self.dt_bias = self.norm_weight = None

    @property
    def channels(self) -> int:
        return 2 * self.G * self.dk + self.H * self.dv

    def cache_need(self):
        return SeveralNeeds((StateNeed((self.H, self.dk, self.dv), torch.float32), StateNeed((self.taps, self.channels), torch.float32)))

    def _common_weights(self, decays: int) -> dict:
        """decays: how many numbers of decay a token has."""
        n, H, G, dk, dv, D = self.names, self.H, self.G, self.dk, self.dv, self.D
        return {n["q"]: WeightSpec((G * dk, D)), n["k"]: WeightSpec((G * dk, D)), n["v"]: WeightSpec((H * dv, D)),
                n["q_conv"]: WeightSpec((G * dk, self.taps), init=("uniform", -0.5, 0.5)),
                n["k_conv"]: WeightSpec((G * dk, self.taps), init=("uniform", -0.5, 0.5)),
                n["v_conv"]: WeightSpec((H * dv, self.taps), init=("uniform", -0.5, 0.5)),
                n["b"]: WeightSpec((H, D)), n["A_log"]: WeightSpec((H,), init=("uniform", -1.0, 1.0), full_precision=True),
                n["dt_bias"]: WeightSpec((decays,), init=("uniform", -6.0, -1.0), full_precision=True),
                n["norm"]: WeightSpec((dv,), init="gain", full_precision=True), n["o"]: WeightSpec((D, H * dv))}

    def _load_common(self, tensors, inputs: tuple) -> list:
        """Everything but the input product, whose rows (the tensors named by `inputs`, of one dtype) are returned."""
        n = self.names
        rows = [tensors[n[k]] for k in inputs]
        if len({r.dtype for r in rows}) > 1:
            rows = [r.to(torch.float32) for r in rows]
        self.w_o = linear.LinearWeight(tensors[n["o"]])
        conv = [tensors[n[k + "_conv"]].to(torch.float32) for k in ("q", "k", "v")]
        self.taps_w = torch.cat(conv, dim=0).t().contiguous()
        self.rate = torch.exp(tensors[n["A_log"]].to(torch.float32)).contiguous()
        self.dt_bias = tensors[n["dt_bias"]].to(torch.float32).contiguous()
        self.norm_weight = tensors[n["norm"]].to(torch.float32).contiguous()
        return rows

    def _input_product(self, rows: list) -> None:
        """All input projections as one product, its width in whole eights."""
        width = sum(r.shape[0] for r in rows)
        self.w_in = linear.LinearWeight(torch.cat([*rows, rows[0].new_zeros((-width % 8, self.D))], dim=0))

    def _project(self, out, residual):
        if residual is None:
            return linear.linear(out, self.w_o, torch.float32)
        linear.linear(out, self.w_o, self.runtime.act_dtype, residual=residual)
        return None


@register_part("mixer", "head_delta")
class HeadDelta(DeltaRule):
    """One decay per head: prompts in chunks of 64 tokens (csrc/head_delta.cu), single tokens in one kernel (csrc/delta.cu)."""
    kernel_libraries = ("head_delta", "delta")

    def __init__(self, runtime: Runtime, hidden_size: int, n_heads: int, key_dim: int, value_dim: int, taps: int, eps: float,
                 n_kv_heads: int | None = None, names: dict | None = None):
        super().__init__(runtime, hidden_size, n_heads, key_dim, value_dim, taps, eps, n_kv_heads,
                         ("q", "k", "v", "b", "A_log", "a", "dt_bias", "g", "norm", "o"), names, 256, "head_delta")

    def weights(self):
        n, H, dv, D = self.names, self.H, self.dv, self.D
        return {**self._common_weights(H), n["a"]: WeightSpec((H, D)), n["g"]: WeightSpec((H * dv, D))}

    def load(self, tensors):
        self._input_product(self._load_common(tensors, ("q", "k", "v", "g", "b", "a")))
        self.g_off = self.channels
        self.b_off = self.g_off + self.H * self.dv
        self.a_off = self.b_off + self.H

    def forward(self, h, ctx: StepContext, cache_view, residual, writes_cache: bool = True):
        state, ring = cache_view
        rows = linear.linear(h, self.w_in, torch.float32)
        before = (rows, self.b_off, self.a_off, self.g_off, self.taps_w, ring, self.dt_bias, self.rate, state, ctx.cu_rows, ctx.slots,
                  ctx.tok_pos, self.norm_weight, self.eps, self.runtime.act_dtype, ctx.B)
        sizes = (self.H, self.G, self.dk, self.dv, self.dk ** -0.5, UNIT_EPS)
        out = ops.head_delta_single(*before, *sizes) if ctx.decode else ops.head_delta_prompt(*before, ctx.max_new, *sizes)
        return self._project(out, residual)


@register_part("mixer", "channel_delta")
class ChannelDelta(DeltaRule):
    kernel_libraries = ("delta", "post_norm", "recurrent")

    def __init__(self, runtime: Runtime, hidden_size: int, n_heads: int, key_dim: int, value_dim: int, taps: int, eps: float,
                 n_kv_heads: int | None = None, rank: int | None = None, gate_rank: int | None = None, names: dict | None = None):
        """rank, gate_rank: the inner sizes of the decays' and the gate's two products; None: whatever the stored tensors have."""
        super().__init__(runtime, hidden_size, n_heads, key_dim, value_dim, taps, eps, n_kv_heads,
                         ("q", "k", "v", "b", "A_log", "a1", "a2", "dt_bias", "g1", "g2", "norm", "o"), names, 4096, "channel_delta")
        self.rank = -1 if rank is None else int(rank)
        self.gate_rank = -1 if gate_rank is None else int(gate_rank)
        self.w_z = self.w_gate = None                 # second products for many rows
        self.a2 = self.g2 = None                      # the same weights for single rows
        self.head_weight = None
        self.ra = self.rg = 0

    def weights(self):
        n, H, dk, dv, D = self.names, self.H, self.dk, self.dv, self.D
        return {**self._common_weights(H * dk), n["a1"]: WeightSpec((self.rank, D)), n["a2"]: WeightSpec((H * dk, self.rank)),
                n["g1"]: WeightSpec((self.gate_rank, D)), n["g2"]: WeightSpec((H * dv, self.gate_rank))}

    def load(self, tensors):
        n = self.names
        # q, k, v, the step sizes and both inner products in one product.
        rows = self._load_common(tensors, ("q", "k", "v", "b", "a1", "g1"))
        self._input_product(rows)
        self.ra, self.rg = rows[4].shape[0], rows[5].shape[0]
        self.b_off = self.channels
        self.a_off = self.b_off + self.H
        self.g_off = self.a_off + self.ra
        self.a2, self.g2 = self._padded(tensors[n["a2"]], self.ra, "a"), self._padded(tensors[n["g2"]], self.rg, "g")
        if self.a2.dtype != self.g2.dtype:
            self.a2, self.g2 = self.a2.to(torch.float32), self.g2.to(torch.float32)
        self.narrow = self.runtime.act_dtype == torch.bfloat16 and self.a2.dtype == torch.bfloat16
        self.w_z = linear.LinearWeight(torch.cat([self.a2, self.a2], dim=1) if self.narrow else self.a2)
        self.w_gate = linear.LinearWeight(self.g2)
        self.head_weight = self.norm_weight.repeat(self.H).contiguous()

    def _padded(self, w, inner: int, which: str):
        """A second product's weight with its inner size in whole eights (zeros behind it)."""
        if w.shape[1] != inner:
            raise ValueError(f"channel_delta: {self.names[which + '1']} has {inner} rows, {self.names[which + '2']} {w.shape[1]} columns")
        return torch.cat([w, w.new_zeros((w.shape[0], -inner % 8))], dim=1).contiguous()

    def forward(self, h, ctx: StepContext, cache_view, residual, writes_cache: bool = True):
        H, G, dk, dv = self.H, self.G, self.dk, self.dv
        act = self.runtime.act_dtype
        state, ring = cache_view
        rows = linear.linear(h, self.w_in, torch.float32)
        if ctx.decode:
            out = ops.delta_single(rows, self.b_off, self.taps_w, ring, self.dt_bias, self.rate, state, ctx.cu_rows, ctx.slots, ctx.tok_pos,
                                   self.a_off, self.ra, self.a2, self.g_off, self.rg, self.g2, self.norm_weight, self.eps, act, ctx.B,
                                   H, G, dk, dv, dk ** -0.5, UNIT_EPS)
        else:
            inner = torch.bfloat16 if self.narrow else torch.float32
            z = linear.linear(ops.take_columns(rows, self.a_off, self.ra, self.a2.shape[1], inner, split=self.narrow), self.w_z, torch.float32)
            gate = linear.linear(ops.take_columns(rows, self.g_off, self.rg, self.g2.shape[1], inner), self.w_gate, act)
            raw = ops.delta_prompt(rows, self.b_off, self.taps_w, ring, z, self.dt_bias, self.rate, state, ctx.cu_rows, ctx.slots,
                                   ctx.tok_pos, ctx.B, ctx.max_new, H, G, dk, dv, dk ** -0.5, UNIT_EPS)
            out = ops.head_norm_gate(raw, dv, self.eps, act, weight=self.head_weight, gate=gate, act="sigmoid")
        return self._project(out, residual)
