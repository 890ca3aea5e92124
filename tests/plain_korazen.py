"""Plain, slow Korazen decoder: the oracle that the engine tests of this design compare with.

Whole sequences, no cache, no batching, one function for each mechanism, float64 by
default, a loop over positions for everything recurrent.  It shares no code with the
product: config.json is read as a plain dict, safetensors with its own few lines, and
every formula is written out here.

The design, in this file's notation (x: the residual stream, which the sublayers read as it
is; t: a position counted from 0; rms(x) = sqrt(mean(x^2) + eps)):

  embedding     x = E[tok] / rms(E[tok]) * w
  layer         x += norm1(mixer(x));  x += norm2(ffn(x))   (ffn may be absent), norm(y) = y / rms(y) * w
  delta rule    q, k (key heads x dim), v (heads x vdim): each channel through a causal convolution over time and
                silu; q and k over sqrt(sum(x^2) + 1e-6) per head, q times dim^-1/2;
                b = sigmoid(W_b x) per head; a = exp(-exp(A) softplus(W_a2 W_a1 x + c)) per head and key channel;
                S' = diag(a_t) S_(t-1);  u = b_t (v_t - S'^T k_t);  S_t = S' + k_t u^T;  o_t = S_t^T q_t;
                each head's o / rms(o) * w (one w for all heads) * sigmoid(W_g2 W_g1 x);  W_o
  two sides     (L / rms(L) * w_l + R / rms(R) * w_r) / 2, both sides reading x
  left side     grouped softmax attention with biases on q, k, v and the output; q and k over their root mean square
                per head times a weight of the head's size; the first r dimensions rotated in pairs (i, i + r/2);
                position t sees j <= t of its own block of n positions; heads times sigmoid(W_g x); W_o
  right side    S_t = d S_(t-1) + k_t v_t^T, o_t = S_t^T q_t with silu on q, k and v and a fixed d per head; all
                heads together over their root mean square times a weight, times sigmoid(W_g x); W_o
  ffn           g = min(W_gate x, m), u = clamp(W_up x, -m, m);  W_down (g sigmoid(1.702 g) (u + 1))
  output        final norm, logits = W_head x times a constant
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import torch

_ST = {"F32": torch.float32, "BF16": torch.bfloat16, "F16": torch.float16, "I32": torch.int32, "I64": torch.int64,
       "F64": torch.float64}


def read_safetensors(path) -> dict[str, torch.Tensor]:
    raw = Path(path).read_bytes()
    (n,) = struct.unpack("<Q", raw[:8])
    header = json.loads(raw[8:8 + n])
    out = {}
    for name, info in header.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        dt = _ST[info["dtype"]]
        t = torch.frombuffer(bytearray(raw[8 + n + lo:8 + n + hi]), dtype=dt) if hi > lo else torch.empty(0, dtype=dt)
        out[name] = t.reshape(info["shape"]).clone()
    return out


def load_folder(folder):
    folder = Path(folder)
    return json.loads((folder / "config.json").read_text()), read_safetensors(folder / "model.safetensors")


# --------------------------------------------------------------------------- small pieces

_STORAGE = None        # set by forward(storage=...): the dtype in which activations are kept between operations
_NOISE = None          # set by forward(noise=...): (relative size, generator)
_MARGINS = None        # set by forward(margins=...): receives how firmly every position of a delta-rule layer reads its state


def _st(x: torch.Tensor) -> torch.Tensor:
    """What a tensor looks like after it was stored in the storage dtype between two operations, or moved as much by chance."""
    if _NOISE is not None:
        size, gen = _NOISE
        x = x * (1.0 + size * (2.0 * torch.rand(x.shape, generator=gen, dtype=x.dtype) - 1.0))
    return x if _STORAGE is None else x.to(_STORAGE).to(x.dtype)


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit_length(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def sigmoid(z: torch.Tensor) -> torch.Tensor:
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rotate_halves(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: pairs (i, i + dims/2) of the first dims dimensions turn by t * base^(-2i/dims) at position t."""
    dims, base = rot["dims"], float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None, None] * f
    c, s = torch.cos(a).to(x.dtype), torch.sin(a).to(x.dtype)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=2)


def causal_conv_silu(z: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """z [T, channels], taps [channels, n]: silu(sum_j taps[:, j] z_(t - n + 1 + j)), rows before the first one zero."""
    T, n = z.shape[0], taps.shape[1]
    out = torch.zeros_like(z)
    for j in range(n):
        back = n - 1 - j                       # tap j looks this many positions back
        out[back:] += taps[:, j] * z[:max(T - back, 0)]
    return silu(out)


# --------------------------------------------------------------------------- gated delta rule

def delta_inputs(h: torch.Tensor, w: dict, m: dict):
    """q, k [T, heads, dim] (key heads repeated), v [T, heads, vdim], b [T, heads], a [T, heads, dim]."""
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _st(causal_conv_silu(_st(h @ w["q"].T), w["q.conv"])).reshape(T, G, dim)
    k = _st(causal_conv_silu(_st(h @ w["k"].T), w["k.conv"])).reshape(T, G, dim)
    v = _st(causal_conv_silu(_st(h @ w["v"].T), w["v.conv"])).reshape(T, H, vdim)
    q, k = unit_length(q) * dim ** -0.5, unit_length(k)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    b = sigmoid(h @ w["b"].T)
    z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
    a = torch.exp(-torch.exp(w["A_log"])[None, :, None] * softplus(z).reshape(T, H, dim))
    return q, k, v, b, a


def delta_rule(q, k, v, b, a, state: list | None = None) -> torch.Tensor:
    """o [T, heads, vdim], token by token."""
    T, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    margins = torch.zeros(T, dtype=torch.float64)
    for t in range(T):
        S = a[t][:, :, None] * S
        u = b[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        if _MARGINS is not None:
            whole = torch.einsum("hdv,hd->hv", S.abs(), q[t].abs())
            margins[t] = float((o[t].norm(dim=1) / whole.norm(dim=1).clamp_min(1e-30)).min())
    if _MARGINS is not None:
        _MARGINS.append(margins)
    if state is not None:
        state.append(S)
    return o


def channel_delta(h: torch.Tensor, w: dict, m: dict, eps: float, state: list | None = None) -> torch.Tensor:
    o = delta_rule(*delta_inputs(h, w, m), state=state)
    o = (unit_rms(o, eps) * w["norm"]).reshape(h.shape[0], m["heads"] * m["vdim"])
    return _st(o * sigmoid(_st(_st(h @ w["g1"].T) @ w["g2"].T))) @ w["o"].T


# --------------------------------------------------------------------------- the two-sided mixer

def visible(i: int, j: int, m: dict) -> bool:
    size = (m.get("mask") or {}).get("size")
    return j <= i and (size is None or i // size == j // size)      # blocks counted from the sequence's first position


def block_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dim, vdim = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w["q"].T + w["q.b"]).reshape(T, H, dim), eps) * w["q.norm"]
    k = unit_rms((h @ w["k"].T + w["k.b"]).reshape(T, G, dim), eps) * w["k.norm"]
    v = _st(h @ w["v"].T + w["v.b"]).reshape(T, G, vdim)
    if m.get("rot"):
        q, k = rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"])
    q, k = _st(q), _st(k)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for t in range(T):
        keys = [j for j in range(t + 1) if visible(t, j, m)]
        kk, vv = k[keys].repeat_interleave(H // G, dim=1), v[keys].repeat_interleave(H // G, dim=1)
        s = torch.einsum("jhd,hd->hj", kk, q[t]) * m["scale"]
        e = torch.exp(s - s.max(dim=1, keepdim=True).values)
        out[t] = torch.einsum("hj,jhv->hv", e / e.sum(dim=1, keepdim=True), vv)
    out = _st(out.reshape(T, H * vdim)) * sigmoid(_st(h @ w["g"].T))
    return _st(out) @ w["o"].T + w["o.b"]


def fixed_decay_attention(h: torch.Tensor, w: dict, m: dict, eps: float, state: list | None = None) -> torch.Tensor:
    T, H, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(_st(h @ w["q"].T)).reshape(T, H, dim)
    k = silu(_st(h @ w["k"].T)).reshape(T, H, dim)
    v = silu(_st(h @ w["v"].T)).reshape(T, H, vdim)
    d = torch.tensor(m["decay"], dtype=torch.float64).to(h.dtype)[:, None, None]
    S = torch.zeros(H, dim, vdim, dtype=h.dtype)
    o = torch.zeros(T, H, vdim, dtype=h.dtype)
    for t in range(T):
        S = d * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
    if state is not None:
        state.append(S)
    o = unit_rms(o.reshape(T, H * vdim), eps) * w["norm"] * sigmoid(_st(h @ w["g"].T))
    return _st(o) @ w["o"].T


def two_sides(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    left = block_attention(h, _sub(w, "left."), m["left"], eps)
    right = fixed_decay_attention(h, _sub(w, "right."), m["right"], eps)
    return 0.5 * (unit_rms(left, eps) * w["left.out"] + unit_rms(right, eps) * w["right.out"])


# --------------------------------------------------------------------------- feed-forward

def clamped_ffn(h: torch.Tensor, w: dict, limit: float) -> torch.Tensor:
    g = torch.clamp(_st(h @ w["gate"].T), max=limit)
    u = torch.clamp(_st(h @ w["up"].T), min=-limit, max=limit)
    return _st(g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


# --------------------------------------------------------------------------- the model

def _sub(weights: dict, prefix: str) -> dict:
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def forward(cfg: dict, weights: dict, tokens, dtype=torch.float64, storage=None, layers_out: list | None = None,
            noise: tuple | None = None, margins: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  storage: the dtype activations are kept in between operations (None: dtype).
    layers_out: receives the residual stream after every layer.  noise = (size, seed): what is stored between operations is
    moved by a relative amount drawn from +-size.  margins: receives for every delta-rule layer how far each position's
    weakest read-out is from cancelling, |S^T q| over |S|^T |q|."""
    global _STORAGE, _NOISE, _MARGINS
    _STORAGE, _MARGINS = storage, margins
    _NOISE = (noise[0], torch.Generator().manual_seed(noise[1])) if noise is not None else None
    try:
        eps = cfg["norm"]["eps"]
        W = {n: t.to(dtype) for n, t in weights.items()}
        x = unit_rms(W["embed"][torch.tensor(list(tokens))], eps) * W["embed.norm"]
        for i, layer in enumerate(cfg["layers"]):
            w = _sub(W, f"l{i}.")
            mixer = channel_delta if layer["type"] == "channel_delta" else two_sides
            x = x + unit_rms(mixer(_st(x), _sub(w, "mix."), layer["mixer"], eps), eps) * w["norm1"]
            if layer.get("mlp"):
                x = x + unit_rms(clamped_ffn(_st(x), _sub(w, "mlp."), layer["mlp"]["limit"]), eps) * w["norm2"]
            if layers_out is not None:
                layers_out.append(x.clone())
        return _st(unit_rms(x, eps) * W["final.norm"]) @ W["head"].T * cfg["logit_scale"]
    finally:
        _STORAGE = _NOISE = _MARGINS = None


def greedy(cfg: dict, weights: dict, prompt, n_new: int) -> list[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
