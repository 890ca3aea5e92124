"""Attention over the paged cache: the choice of kernel, and the work lists that the prompt kernels read."""
from __future__ import annotations

import numpy as np
import torch

from . import ops

USE_TC_PREFILL = True        # head_dim 64 and 128: prefill attention on tcgen05 instead of mma.sync
BALANCED_DECODE = True       # steps of single tokens: the keys of all sequences cut into equal shares (else equal slices per sequence)
MAX_SPLITS = 32
KEYS_PER_SPLIT = 128         # a slice shorter than this is not worth a block of its own

def resident_blocks(device, hd: int = 128) -> int:
    """Blocks of the decode kernel that run at a time: one (8 warps, ~200 KB of key/value rings) per SM,
    two where the rings are half as large (hd, the larger of a head's key and value sizes, up to 64)."""
    return ops.sm_count(device) * (2 if hd <= 64 else 1)


def decode_splits(n_tokens: int, Hkv: int, group_tiles: int, max_kv: int, resident: int) -> int:
    """How many slices to cut each sequence's keys into: as many as still run in one wave."""
    blocks = max(1, n_tokens * Hkv * group_tiles)
    return max(1, min(resident // blocks, MAX_SPLITS, -(-max_kv // KEYS_PER_SPLIT)))


# ------------------------------------------------------------------ work lists of the prompt kernels
def query_blocks(size: int):
    """Builder of the work list of a prompt kernel whose blocks take `size` query rows: blocks of at most
    `size` consecutive rows of one sequence, as int32 [4, n] = (sequence, first row, rows, first position),
    the blocks with the most keys first.  A step of one token per sequence needs none."""
    def build(step) -> np.ndarray:
        if step.max_new == 1:
            return np.zeros(0, dtype=np.int32)
        qb = [(b, step.cu[b] + r, min(size, n - r), p + r)
              for b, (p, n) in enumerate(zip(step.past, step.new)) for r in range(0, n, size)]
        qb.sort(key=lambda e: -e[3])
        return np.asarray(qb, dtype=np.int32).reshape(-1, 4).T.copy()
    return build


# ------------------------------------------------------------------ work list of the decode kernel
MIN_PART_TILES = KEYS_PER_SPLIT // 16      # the same floor in the kernel's 16-key tiles
DECODE_TILE = 16


def decode_teams(B: int, Hkv: int, group_tiles: int, resident: int) -> int:
    """Room in the work list of a batch of B tokens: the teams of blocks (one block per kv head and row
    tile each) that run as one wave, and at least one team per token.  Not more: with parts for one and a
    half to three waves, steps of sequences of unequal lengths ran 0 to 12 % slower (3B and 8B layer sizes,
    batches of 8 to 32), because a block of a later wave starts its loads from nothing."""
    return min(max(B, resident // max(1, Hkv * group_tiles)), 65535)


def decode_work_size(B: int, teams: int) -> int:
    return teams + 1 + 5 * teams


def cut_decode_work(positions, window: int, teams: int, max_parts: int = MAX_SPLITS, keep_first: int = 0, chunk: int = 0) -> np.ndarray:
    """The decode kernel's work list for tokens at these positions: every token's keys cut into parts of
    nearly the same length for all tokens, as short as `teams` parts in all allow, so that a long sequence
    gets more parts than a short one and the blocks finish together (with the same number of slices for
    every sequence, the blocks of the longest would still run when all others are done).  The longest
    parts come first.  int32 [teams + 1 + 5 * teams]: for each team the offset of its segments (here one
    each, or none), then (token, first tile, last tile + 1, part, parts of the token) per segment, in the
    kernel's 16-key tiles counted from the first one the token sees (its window's first tile; with
    `keep_first`, the tiles of the kept first positions that lie ahead of the window are counted before the
    window's).  With `chunk` n instead of a window, a token's first tile is the one that holds the first position of
    its block of n positions.  No part is shorter than MIN_PART_TILES unless it is a whole token, and no token gets more
    than max_parts."""
    pos = np.asarray(positions, dtype=np.int64)
    B = len(pos)
    if teams < B:
        raise ValueError(f"{B} tokens need at least as many teams, not {teams}")
    if chunk > 0:
        first = (pos - pos % chunk) // DECODE_TILE
    else:
        first = np.where((window > 0) & (pos >= window), pos - window + 1, 0) // DECODE_TILE
    if window > 0 and keep_first > 0:
        first = first - np.minimum(-(-keep_first // DECODE_TILE), first)       # the kept tiles count as well
    tiles = pos // DECODE_TILE + 1 - first
    most = np.minimum(max_parts, np.maximum(1, tiles // MIN_PART_TILES))       # parts a token may have
    n = np.ones(B, dtype=np.int64)
    if teams > B and most.max() > 1:
        # The best common length is some token's length over some count of parts: try them all at once.
        counts = np.arange(1, min(max_parts, teams - B + 1) + 1)
        lengths = np.unique(-(-tiles[:, None] // counts[None, :]))
        need = np.minimum(-(-tiles[None, :] // lengths[:, None]), most[None, :])
        fits = need.sum(axis=1) <= teams
        n = need[np.argmax(fits)]              # lengths ascend: the first that fits is the shortest
    tok = np.repeat(np.arange(B), n)
    part = np.arange(len(tok)) - np.repeat(np.cumsum(n) - n, n)
    lo, hi = part * tiles[tok] // n[tok], (part + 1) * tiles[tok] // n[tok]
    order = np.argsort(lo - hi, kind="stable")
    out = np.zeros(decode_work_size(B, teams), dtype=np.int32)
    out[:teams + 1] = np.minimum(np.arange(teams + 1), len(tok))
    seg = out[teams + 1:teams + 1 + 5 * len(tok)].reshape(-1, 5)
    seg[:, 0], seg[:, 1], seg[:, 2], seg[:, 3], seg[:, 4] = tok[order], lo[order], hi[order], part[order], n[tok][order]
    return out


def decode_work(H: int, Hkv: int, window: int | None, device, hd: int = 128, keep_first: int = 0, chunk: int | None = None):
    """Builder of the decode kernel's work list for attention of these head counts, this window (or these blocks of
    positions) and these kept first positions: empty for a step with prompts."""
    group_tiles = -(-(H // Hkv) // 16)

    def build(step) -> np.ndarray:
        if step.max_new != 1:
            return np.zeros(0, dtype=np.int32)
        return cut_decode_work(np.asarray(step.past), int(window or 0),
                               decode_teams(step.B, Hkv, group_tiles, resident_blocks(device, hd)),
                               keep_first=int(keep_first or 0), chunk=int(chunk or 0))
    return build


def decode_work_name(H: int, Hkv: int, window: int | None, keep_first: int = 0, chunk: int | None = None) -> str:
    kept = int(keep_first or 0) if window else 0
    return f"decode_work:{H}:{Hkv}:{ops.span(window, chunk)}" + (f":{kept}" if kept else "")


PREFILL_LISTS = {"query_blocks64": query_blocks(64), "query_blocks128": query_blocks(128)}


def _mma_sizes(hd: int, vd: int | None) -> bool:
    """Head sizes that the mma.sync kernels take: keys of whole sixteens up to 128, values of whole eights up to 256."""
    return hd % 16 == 0 and hd <= 128 and (vd is None or (vd % 8 == 0 and vd <= 256))


def prefill_kernel(dtype: torch.dtype, hd: int, page_size: int = 64, vd: int | None = None) -> str | None:
    """Which prompt kernel takes queries of this dtype, head size and value size (None: the head's): "tc" (tcgen05),
    "mma" (mma.sync), or None (the plain kernel)."""
    if dtype != torch.bfloat16 or page_size != 64:
        return None
    if USE_TC_PREFILL and hd in (64, 128) and vd in (None, hd):
        return "tc"
    return "mma" if _mma_sizes(hd, vd) else None


def decode_kernel(dtype: torch.dtype, hd: int, vd: int | None = None) -> bool:
    """Whether single tokens of this dtype, head size and value size go to the split decode kernel."""
    return dtype == torch.bfloat16 and _mma_sizes(hd, vd)


def step_needs(dtype: torch.dtype, hd: int, H: int | None = None, Hkv: int | None = None, window: int | None = None,
               device=None, keep_first: int = 0, chunk: int | None = None, vd: int | None = None) -> dict:
    """The work lists that attention of this dtype and head size reads: the query blocks of steps with
    prompts, and (when the head counts are given) the balanced segments of steps of single tokens."""
    kind = prefill_kernel(dtype, hd, vd=vd)
    name = {"tc": "query_blocks128", "mma": "query_blocks64"}.get(kind)
    needs = {name: PREFILL_LISTS[name]} if name else {}
    if H is not None and Hkv and BALANCED_DECODE and decode_kernel(dtype, hd, vd):
        needs[decode_work_name(H, Hkv, window, keep_first, chunk)] = decode_work(H, Hkv, window, device, max(hd, vd or hd), keep_first, chunk)
    return needs


def _blocks(ctx, name):
    flat = ctx.extra.get(name)
    if flat is None or flat.numel() == 0:
        return None
    return tuple(flat.view(4, -1))


def attention(qkv, cache_view, ctx, H, Hkv, hd, scale, window, next_w=None, vd=None, sink=None, gate=None, softcap=None,
              keep_first=0, chunk=None, gate_per_head=False, slope=None):
    """Rows of qkv hold q in their left H*hd columns.  Returns [T, H*vd].  next_w: the weights the
    stream reads after the attention (the decode kernel asks for their first bytes as it ends).
    vd: size of a value head (default hd); sink: float32 [H], one more term of each head's softmax
    denominator; gate: [T, H*vd] whose sigmoid multiplies the output; softcap c: score <- c tanh(score / c);
    keep_first n: with a window, a sequence's first n positions stay visible.  chunk n (instead of a window): a position
    sees only its own block of n positions.  gate_per_head: the gate is [T, H], one number for a head's values.
    slope: float32 [H], a score loses slope[h] times the distance to its key (after the scale and the cap)."""
    vd = vd or hd
    keep_first = int(keep_first or 0) if window else 0
    out = _attention(qkv, cache_view, ctx, H, Hkv, hd, scale, window, next_w, sink, gate, softcap, keep_first, chunk, vd, slope)
    if gate is not None and out is not None:
        # The tensor-core kernels leave the gate to a kernel of its own.
        return ops.gate_mul(out, gate, "sigmoid", group=vd if gate_per_head else 1)
    return out if out is not None else general_attention(qkv, cache_view, ctx, H, Hkv, hd, vd, scale, window, sink, gate,
                                                         softcap, keep_first, chunk, gate_per_head, slope)


def _attention(qkv, cache_view, ctx, H, Hkv, hd, scale, window, next_w, sink, gate, softcap, keep_first, chunk, vd, slope):
    """The tensor-core kernels where they take the sizes; None where only the plain kernel does and a gate
    is to be applied or values have a size of their own (the plain kernel does both itself)."""
    aligned = qkv.stride(0) % 8 == 0 and qkv.data_ptr() % 16 == 0
    more = dict(sink=sink, softcap=softcap, keep_first=keep_first, slope=slope)
    mask = ops.span(window, chunk)          # the kernels take a window as w and blocks of n positions as -n
    if not ctx.decode and aligned:
        kind = prefill_kernel(qkv.dtype, hd, cache_view.page_size, vd)
        if kind == "tc":
            blocks = _blocks(ctx, "query_blocks128")
            if blocks is not None:
                return ops.attn_prefill_tc(qkv, cache_view.k_pages, cache_view.v_pages, cache_view.page_table, ctx.slots,
                                           ctx.kv_len, blocks, H, Hkv, hd, cache_view.page_size, scale, mask, **more)
            kind = "mma" if "query_blocks64" in ctx.extra else None
        if kind == "mma":
            blocks = _blocks(ctx, "query_blocks64")
            if blocks is not None:
                return ops.attn_prefill(qkv, cache_view.k_pages, cache_view.v_pages, cache_view.page_table, ctx.slots,
                                        ctx.kv_len, blocks, H, Hkv, hd, cache_view.page_size, scale, mask, vd=vd, **more)
    if ctx.decode and aligned and decode_kernel(qkv.dtype, hd, vd) and cache_view.page_size % 16 == 0:
        work = ctx.extra.get(decode_work_name(H, Hkv, window, keep_first, chunk))
        if work is not None and work.numel():
            teams = decode_teams(ctx.T, Hkv, -(-(H // Hkv) // 16), resident_blocks(qkv.device, max(hd, vd)))
            if work.numel() == decode_work_size(ctx.T, teams):
                return ops.attn_decode(qkv, cache_view.k_pages, cache_view.v_pages, cache_view.page_table, ctx.tok_pos,
                                       ctx.tok_seq, ctx.slots, H, Hkv, hd, cache_view.page_size, scale, mask,
                                       min(MAX_SPLITS, teams), next_w=next_w, early_loads=True, work=work, teams=teams,
                                       vd=vd, **more)
        n_splits = decode_splits(ctx.T, Hkv, -(-(H // Hkv) // 16), ctx.max_kv, resident_blocks(qkv.device, max(hd, vd)))
        return ops.attn_decode(qkv, cache_view.k_pages, cache_view.v_pages, cache_view.page_table, ctx.tok_pos,
                               ctx.tok_seq, ctx.slots, H, Hkv, hd, cache_view.page_size, scale, mask, n_splits,
                               next_w=next_w, early_loads=True, vd=vd, **more)      # a decode step: one new token per sequence
    if gate is not None or vd != hd:
        return None
    return ops.attention_plain(qkv, cache_view.k_pages, cache_view.v_pages, cache_view.page_table, ctx.tok_pos,
                               ctx.tok_seq, ctx.slots, H, Hkv, hd, cache_view.page_size, scale, window, sink=sink,
                               softcap=softcap, keep_first=keep_first, chunk=chunk, slope=slope)


def general_attention(qkv, cache_view, ctx, H, Hkv, hd, vd, scale, window, sink, gate, softcap=None, keep_first=0, chunk=None,
                      gate_per_head=False, slope=None):
    """Attention through the plain kernel, which takes every option: a sink, a gate (per value or per head), values of
    another size than the keys, capped scores, kept first positions, blocks of positions."""
    return ops.attention_plain(qkv, cache_view.k_pages, cache_view.v_pages, cache_view.page_table, ctx.tok_pos,
                               ctx.tok_seq, ctx.slots, H, Hkv, hd, cache_view.page_size, scale, window, vd=vd,
                               sink=sink, gate=gate, softcap=softcap, keep_first=keep_first, chunk=chunk,
                               gate_per_head=gate_per_head, slope=slope)
