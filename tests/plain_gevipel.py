"""Plain, slow Gevipel decoder: the oracle that the engine tests of this design compare with.

Whole sequences, no cache, no batching, one function for each mechanism, float64 by
default, a loop over positions for everything recurrent.  It shares no code with the
product: config.json is read as a plain dict, safetensors with its own few lines, and
every formula is written out here.

The design, in this file's notation (x: the residual stream; t: a position counted from 0;
LN(x) = (x - mean) / sqrt(var + eps) * g + b; rms(x) = sqrt(mean(x^2) + eps)):

  embedding     e = s E[tok];  x = e
  layer         x += m LN1b(mixer(LN1(x)));  x += m LN2b(ffn(LN2(x)))   (ffn may be absent)
  repeats       a stretch of layers runs several times; ahead of every pass but the first x += e
  delta         q, k (key heads x dim), v (heads x vdim): each channel through a causal convolution over time and
                silu; q and k over sqrt(sum(x^2) + 1e-6) per head, q times dim^-1/2;
                b = sigmoid(W_b h), a = exp(-exp(A) softplus(W_a h + c)), one number per head each;
                S' = a_t S_(t-1);  u = b_t (v_t - S'^T k_t);  S_t = S' + k_t u^T;  o_t = S_t^T q_t;
                each head's o / rms(o) * w (one w for all heads) * silu(W_g h);  W_o
  attention     grouped softmax attention without rotation whose values are the keys as projected; q and k over their
                root mean square per head times a weight of the head's size; q times 1 + c ln(floor((t + 1) / n) + 1);
                score = scale q . k - 2^(-8 (head + 1) / heads) (t - j) for 0 <= t - j < window;  W_o
  latent        q = W_q h, per head [unrotated | rotated]; [c' | r] = W_dkv h, c = c' / rms(c') * w; keys W_uk c, values
                W_uv c per head, r rotated and shared by all heads; pairs (2i, 2i + 1) turn by t base^(-2i/dims);
                score = scale (q . k + q_r . r); the softmax denominator holds one more exp(sink_head);  W_o
  ffn           s = softmax(W_router h) over all experts; the `top` largest s + correction are chosen;
                sum of s_e W_down,e relu(W_up,e h)^2 over them
  output        LN, logits = W_head x
"""
from __future__ import annotations

import json
import math
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
_MARGINS = None        # set by forward(margins=...): how firmly every position of a layer does what it does (a list per kind)


def _st(x: torch.Tensor) -> torch.Tensor:
    """What a tensor looks like after it was stored in the storage dtype between two operations, or moved as much by chance."""
    if _NOISE is not None:
        size, gen = _NOISE
        x = x * (1.0 + size * (2.0 * torch.rand(x.shape, generator=gen, dtype=x.dtype) - 1.0))
    return x if _STORAGE is None else x.to(_STORAGE).to(x.dtype)


def layer_norm(x: torch.Tensor, g: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * g + b


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


def rotate_neighbours(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, dim]: pairs (2i, 2i + 1) of the first dims dimensions turn by t * base^(-2i/dims) at position t."""
    dims, base = rot["dims"], float(rot["base"])
    out = x.clone()
    t = torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(dims // 2):
        a = t * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        out[:, :, 2 * i], out[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def causal_conv_silu(z: torch.Tensor, taps: torch.Tensor) -> torch.Tensor:
    """z [T, channels], taps [channels, n]: silu(sum_j taps[:, j] z_(t - n + 1 + j)), rows before the first one zero."""
    T, n = z.shape[0], taps.shape[1]
    out = torch.zeros_like(z)
    for j in range(n):
        back = n - 1 - j                       # tap j looks this many positions back
        out[back:] += taps[:, j] * z[:max(T - back, 0)]
    return silu(out)


# --------------------------------------------------------------------------- gated delta rule, one decay per head

def delta_inputs(h: torch.Tensor, w: dict, m: dict):
    """q, k [T, heads, dim] (key heads repeated), v [T, heads, vdim], b and a [T, heads]."""
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = _st(causal_conv_silu(_st(h @ w["q"].T), w["q.conv"])).reshape(T, G, dim)
    k = _st(causal_conv_silu(_st(h @ w["k"].T), w["k.conv"])).reshape(T, G, dim)
    v = _st(causal_conv_silu(_st(h @ w["v"].T), w["v.conv"])).reshape(T, H, vdim)
    q, k = unit_length(q) * dim ** -0.5, unit_length(k)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    b = sigmoid(h @ w["b"].T)
    a = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    return q, k, v, b, a


def delta_rule(q, k, v, b, a, state: list | None = None) -> torch.Tensor:
    """o [T, heads, vdim], token by token."""
    T, H, dim = q.shape
    S = torch.zeros(H, dim, v.shape[2], dtype=q.dtype)
    o = torch.zeros_like(v)
    firm = torch.zeros(T, dtype=torch.float64)
    for t in range(T):
        S = a[t][:, None, None] * S
        u = b[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = torch.einsum("hdv,hd->hv", S, q[t])
        if _MARGINS is not None:
            whole = torch.einsum("hdv,hd->hv", S.abs(), q[t].abs())
            firm[t] = float((o[t].norm(dim=1) / whole.norm(dim=1).clamp_min(1e-30)).min())
    if _MARGINS is not None:
        _MARGINS["read"].append(firm)
    if state is not None:
        state.append(S)
    return o


def delta(h: torch.Tensor, w: dict, m: dict, eps: float, state: list | None = None) -> torch.Tensor:
    o = delta_rule(*delta_inputs(h, w, m), state=state)
    o = (unit_rms(o, eps) * w["norm"]).reshape(h.shape[0], m["heads"] * m["vdim"])
    return _st(o * silu(_st(h @ w["g"].T))) @ w["o"].T


# --------------------------------------------------------------------------- softmax attention

def slopes(H: int) -> torch.Tensor:
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=torch.float64)


def temperature(T: int, m: dict) -> torch.Tensor:
    qt = m.get("q_temp")
    if not qt:
        return torch.ones(T, dtype=torch.float64)
    return torch.tensor([1.0 + qt["coef"] * math.log(math.floor((t + 1) / qt["every"]) + 1.0) for t in range(T)], dtype=torch.float64)


def softmax_rows(s: torch.Tensor, extra: torch.Tensor | None = None) -> torch.Tensor:
    """s [H, keys]; extra [H]: one more term of each denominator that has no key."""
    top = s.max(dim=1, keepdim=True).values
    if extra is not None:
        top = torch.maximum(top, extra[:, None])
    e = torch.exp(s - top)
    den = e.sum(dim=1, keepdim=True)
    if extra is not None:
        den = den + torch.exp(extra[:, None] - top)
    return e / den


def attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, G, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    size = (m.get("mask") or {}).get("size")
    raw = (h @ w["k"].T).reshape(T, G, dim)
    q = unit_rms((h @ w["q"].T).reshape(T, H, dim), eps) * w["q.norm"]
    q = _st(q * temperature(T, m).to(h.dtype)[:, None, None])
    k = _st(unit_rms(raw, eps) * w["k.norm"]).repeat_interleave(H // G, dim=1)
    v = _st(raw).repeat_interleave(H // G, dim=1)
    slope = slopes(H).to(h.dtype)[:, None]
    out = torch.zeros(T, H, dim, dtype=h.dtype)
    for t in range(T):
        lo = 0 if size is None else max(0, t - size + 1)
        back = torch.arange(t - lo, -1, -1, dtype=h.dtype)                 # t - j
        s = torch.einsum("jhd,hd->hj", k[lo:t + 1], q[t]) * m["scale"] - slope * back
        out[t] = torch.einsum("hj,jhv->hv", softmax_rows(s), v[lo:t + 1])
    return _st(out.reshape(T, H * dim)) @ w["o"].T


def latent_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T, H, dn, dr, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = _st(h @ w["q"].T).reshape(T, H, dn + dr)
    down = h @ w["dkv"].T
    c = _st(unit_rms(down[:, :R], eps) * w["dkv.norm"])
    k = (c @ w["uk"].T).reshape(T, H, dn)
    v = (c @ w["uv"].T).reshape(T, H, dv)
    q_r, r = q[:, :, dn:], down[:, None, R:]
    if dr and m.get("rot"):
        q_r, r = rotate_neighbours(q_r, m["rot"]), rotate_neighbours(r, m["rot"])
    r = _st(r)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        s = torch.einsum("jhd,hd->hj", k[:t + 1], q[t, :, :dn]) + torch.einsum("jd,hd->hj", r[:t + 1, 0], q_r[t])
        out[t] = torch.einsum("hj,jhv->hv", softmax_rows(s * m["scale"], w["sink"]), v[:t + 1])
    return _st(out.reshape(T, H * dv)) @ w["o"].T


MIXERS = {"delta": delta, "attention": attention, "latent_attention": latent_attention}


# --------------------------------------------------------------------------- feed-forward

def route(z: torch.Tensor, correction: torch.Tensor, top: int):
    """Chosen experts (largest choice scores first; the lower number wins a tie), their weights, and by how much the last
    one was chosen ahead of the first that was not."""
    e = torch.exp(z - z.max())
    s = e / e.sum()
    choice = s + correction
    order = sorted(range(z.numel()), key=lambda i: (-float(choice[i]), i))
    gap = float(choice[order[top - 1]] - choice[order[top]]) if z.numel() > top else math.inf
    return order[:top], s[order[:top]], gap


def routed_ffn(h: torch.Tensor, w: dict, mlp: dict) -> torch.Tensor:
    out = torch.zeros_like(h)
    gaps = torch.zeros(h.shape[0], dtype=torch.float64)
    for t in range(h.shape[0]):
        experts, weights, gaps[t] = route(w["router"] @ h[t], w["correction"], mlp["router"]["top"])
        for e, p in zip(experts, weights):
            u = torch.clamp(w[f"e{e}.up"] @ h[t], min=0.0)
            out[t] += p * (w[f"e{e}.down"] @ _st(u * u))
    if _MARGINS is not None:
        _MARGINS["route"].append(gaps)
    return out


# --------------------------------------------------------------------------- the model

def _sub(weights: dict, prefix: str) -> dict:
    return {n[len(prefix):]: t for n, t in weights.items() if n.startswith(prefix)}


def layer_order(cfg: dict) -> list[tuple[int, bool]]:
    """(layer, whether the embedding's output joins the stream right ahead of it) for every run of a layer."""
    n = len(cfg["layers"])
    loop = cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    lo, hi = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(lo)]
    for turn in range(loop["times"]):
        runs += [(i, turn > 0 and i == lo) for i in range(lo, hi)]
    return runs + [(i, False) for i in range(hi, n)]


def new_margins() -> dict:
    return {"read": [], "route": []}


def forward(cfg: dict, weights: dict, tokens, dtype=torch.float64, storage=None, layers_out: list | None = None,
            noise: tuple | None = None, margins: dict | None = None) -> torch.Tensor:
    """Logits [T, vocab] of one sequence.  storage: the dtype activations are kept in between operations (None: dtype).
    layers_out: receives the residual stream after every run of a layer.  noise = (size, seed): what is stored between
    operations is moved by a relative amount drawn from +-size.  margins (see new_margins): receives for every run of a
    delta layer how far each position's weakest read-out is from cancelling, |S^T q| over |S|^T |q| ("read"), and for every
    run of a feed-forward by how much each position's last expert was chosen ("route")."""
    global _STORAGE, _NOISE, _MARGINS
    _STORAGE, _MARGINS = storage, margins
    _NOISE = (noise[0], torch.Generator().manual_seed(noise[1])) if noise is not None else None
    try:
        eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
        W = {n: t.to(dtype) for n, t in weights.items()}
        e = W["embed"][torch.tensor(list(tokens))] * cfg["embedding"]["scale"]
        x = e.clone()
        for i, reenter in layer_order(cfg):
            layer, w = cfg["layers"][i], _sub(W, f"l{i}.")
            if reenter:
                x = x + e
            y = MIXERS[layer["type"]](_st(layer_norm(x, w["norm1"], w["norm1.b"], eps)), _sub(w, "mix."), layer["mixer"], eps)
            x = x + m * layer_norm(y, w["norm1b"], w["norm1b.b"], eps)
            if layer.get("mlp"):
                y = routed_ffn(_st(layer_norm(x, w["norm2"], w["norm2.b"], eps)), _sub(w, "mlp."), layer["mlp"])
                x = x + m * layer_norm(y, w["norm2b"], w["norm2b.b"], eps)
            if layers_out is not None:
                layers_out.append(x.clone())
        return _st(layer_norm(x, W["final.norm"], W["final.norm.b"], eps)) @ W["head"].T
    finally:
        _STORAGE = _NOISE = _MARGINS = None


def greedy(cfg: dict, weights: dict, prompt, n_new: int) -> list[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
