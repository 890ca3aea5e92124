"""Small Gevipel configurations and model folders with random weights, for the tests of this design.

The configurations differ from each other in every size and option: delta heads of 8 to 200 key channels and 5 to 160
values, as many key heads as value heads and fewer, convolutions of 1 to 7 taps; attention with windows of 1, 5, 20, 64, 70
and 100 positions and over all of them, grouped and not, with and without a query temperature, heads of 12 to 128; latent
attention with ranks of 20 to 300, rotated parts of none to 32, values wider and narrower than keys; experts of 12 to 64,
one, some or all of them per token, and layers without; loops of one to three passes anywhere in the list; embedding
scales and multipliers on the branches that are one and that are not; widths and head sizes that are no multiples of 8.
"""
from __future__ import annotations

from pathlib import Path

import numpy as np
import torch

import plain_gevipel


def delta(heads, kv_heads, dim, vdim, conv=4, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def attn(heads, kv_heads, dim, window=None, temp=None, scale=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5 if scale is None else scale}
    if window is not None:
        m["mask"] = {"size": window}
    if temp is not None:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent(heads, dim, rot_dim, vdim, kv_rank, base=1e4, scale=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    if rot_dim:
        m["rot"] = {"dims": rot_dim, "base": base}
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def model(width, vocab, layers, eps=1e-5, loop=None, scale=1.0, mult=1.0):
    out = {"architecture": "Gevipel", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
           "residual_mult": mult, "layers": layers}
    if loop is not None:
        out["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return out


CONFIGS = {
    # one mechanism each
    "only_delta": model(48, 120, [delta(4, 2, 16, 24, conv=4)], scale=1.7),
    "only_delta_even": model(64, 90, [delta(2, 2, 64, 64, conv=3)], mult=0.6),
    "only_delta_wide_keys": model(40, 100, [delta(2, 1, 200, 20, conv=5)], eps=1e-6),
    "only_delta_wide_values": model(40, 90, [delta(2, 2, 24, 160, conv=2)], scale=0.5),
    "only_delta_odd": model(36, 77, [delta(3, 3, 20, 37, conv=7)], mult=1.4),
    "only_delta_no_past": model(32, 80, [delta(6, 2, 8, 5, conv=1)]),
    "only_attention": model(64, 140, [attn(4, 2, 64, window=40, temp=(0.4, 16))], mult=0.5),
    "only_attention_mma": model(48, 110, [attn(6, 3, 48, window=20, temp=(0.2, 50), scale=0.3)], scale=2.0),
    "only_attention_wide": model(64, 100, [attn(2, 2, 128, window=100)]),
    "only_attention_open": model(36, 100, [attn(5, 1, 12, temp=(1.0, 3))], eps=1e-6),
    "only_latent": model(64, 140, [latent(4, 32, 16, 24, 64)], mult=0.7),
    "only_latent_odd": model(36, 90, [latent(3, 20, 12, 28, 36, base=100.0, scale=0.3)], scale=1.3),
    "only_latent_wide": model(64, 90, [latent(5, 16, 32, 64, 304, base=5e5)]),
    "only_latent_still": model(40, 80, [latent(2, 24, 0, 8, 24)]),
    "only_experts": model(32, 90, [attn(2, 1, 16, mlp=moe(8, 3, 24))], mult=0.8),
    "only_experts_all": model(32, 90, [attn(2, 2, 16, mlp=moe(3, 3, 20))]),
    "only_experts_one": model(32, 90, [attn(2, 2, 16, mlp=moe(5, 1, 16))]),
    "only_loop": model(32, 90, [attn(2, 1, 16, window=30, mlp=moe(4, 2, 16)), delta(2, 1, 8, 12)], loop=(0, 2, 3), scale=0.7, mult=0.9),
    "only_loop_once": model(32, 90, [attn(2, 1, 16), latent(2, 8, 8, 8, 16), attn(2, 1, 16)], loop=(1, 2, 1)),
    # whole models
    "mixed": model(64, 200, [
        latent(4, 24, 8, 32, 40, base=1e4, mlp=moe(6, 2, 32)),
        delta(4, 2, 32, 48, conv=4, mlp=moe(5, 3, 24)),
        attn(4, 2, 32, window=64, temp=(0.3, 40), mlp=moe(6, 2, 32)),
        delta(2, 2, 24, 16, conv=3, mlp=None),
        attn(2, 1, 64, window=100, temp=(0.5, 64), mlp=moe(4, 2, 48))], loop=(1, 4, 2), scale=2.5, mult=0.4),
    "odd": model(44, 131, [
        attn(3, 1, 20, window=5, temp=(0.6, 7), mlp=moe(3, 2, 12)),
        latent(3, 12, 4, 20, 20, base=50.0, mlp=None),
        delta(3, 1, 36, 28, conv=5, mlp=moe(5, 2, 20)),
        attn(5, 5, 12, window=1, mlp=None)], eps=1e-6, loop=(2, 4, 3), scale=0.6, mult=1.2),
    "wide": model(128, 300, [
        delta(4, 4, 128, 64, conv=4, mlp=moe(8, 3, 64)),
        attn(4, 2, 128, window=100, temp=(0.2, 100), mlp=moe(8, 2, 40)),
        latent(8, 32, 32, 64, 128, base=1e6, mlp=moe(6, 2, 64)),
        attn(4, 1, 64, window=70, mlp=None),
        delta(2, 1, 64, 128, conv=4, mlp=moe(4, 2, 32))], loop=(0, 3, 2), scale=1.5, mult=0.5),
}


def random_config(rng) -> dict:
    """A configuration whose sizes and options nobody chose."""
    layers = []
    for _ in range(rng.randint(2, 5)):
        experts = rng.randint(2, 7)
        mlp = moe(experts, rng.randint(1, experts), rng.choice([8, 12, 24, 32])) if rng.random() < 0.6 else None
        g = rng.randint(1, 3)
        h = g * rng.randint(1, 3)
        kind = rng.choice(["delta", "attention", "latent"])
        if kind == "delta":
            layers.append(delta(h, g, rng.choice([8, 16, 40, 64]), rng.choice([8, 12, 33, 48]), conv=rng.randint(1, 6), mlp=mlp))
        elif kind == "attention":
            temp = (rng.choice([0.2, 0.7]), rng.choice([4, 30, 64])) if rng.random() < 0.7 else None
            layers.append(attn(h, g, rng.choice([8, 16, 32, 64, 96]), window=rng.choice([None, 3, 17, 64, 90]), temp=temp,
                               scale=rng.choice([None, 0.1, 0.25]), mlp=mlp))
        else:
            layers.append(latent(rng.randint(1, 6), rng.choice([8, 16, 24]), rng.choice([0, 4, 8, 16]), rng.choice([8, 20, 32]),
                                 rng.choice([12, 32, 64, 96]), base=rng.choice([100.0, 1e4, 1e6]), mlp=mlp))
    loop = None
    if rng.random() < 0.7:
        lo = rng.randint(0, len(layers) - 1)
        loop = (lo, rng.randint(lo + 1, len(layers)), rng.randint(1, 3))
    return model(rng.choice([24, 40, 56, 64, 72]), rng.choice([77, 128, 200]), layers, eps=rng.choice([1e-5, 1e-6]), loop=loop,
                 scale=rng.choice([0.5, 1.0, 3.0]), mult=rng.choice([0.3, 0.8, 1.0]))


def make_folder(tmp, name, seed: int = 0, std: float = 0.1, gain_std: float = 0.2, dtype=torch.bfloat16) -> Path:
    """A model folder with random weights, written by the framework's random-weights mode."""
    import longbow_quarrel_b200  # noqa: F401
    from longbow_quarrel_b200 import architectures  # noqa: F401
    from longbow_quarrel_b200.config import architecture_of
    from longbow_quarrel_b200.engine.model import Model
    from longbow_quarrel_b200.parts.base import Runtime
    from longbow_quarrel_b200.weights import write_random_model
    data = CONFIGS[name] if isinstance(name, str) else name
    arch = architecture_of(data)
    cfg = arch.config_from_dict(data)
    table = Model(arch.describe(cfg), Runtime(torch.device("cpu"), torch.float32, 64)).weight_table()
    label = name if isinstance(name, str) else "custom"
    return write_random_model(Path(tmp) / f"gevipel_{label}_{seed}", cfg.to_dict(), table, seed, dtype, std, gain_std)


def rewrite(folder, change) -> None:
    """Change a folder's weights in place: change(weights) edits the dictionary of tensors."""
    from longbow_quarrel_b200.weights import write_safetensors
    weights = plain_gevipel.read_safetensors(Path(folder) / "model.safetensors")
    change(weights)
    write_safetensors(Path(folder) / "model.safetensors", weights, {"format": "pt"})


def tokens(n: int, vocab: int, seed: int) -> list[int]:
    return [int(t) for t in np.random.default_rng(seed).integers(0, vocab, size=n)]


def row_errors(got: np.ndarray, ref: np.ndarray) -> np.ndarray:
    """Per row: root mean square of the difference over the root mean square of the reference row."""
    got, ref = np.asarray(got, np.float64), np.asarray(ref, np.float64)
    assert got.shape == ref.shape, (got.shape, ref.shape)
    assert np.isfinite(got).all(), "non-finite logits"
    return np.sqrt(((got - ref) ** 2).mean(-1)) / np.maximum(np.sqrt((ref ** 2).mean(-1)), 1e-30)


F32_TOL = 2e-5        # the floor of every float32 bound, per row

# What a read-out of the delta rule is of what it would be if nothing in it cancelled, and by how much the last expert was
# chosen: below these, rounding may turn the read-out's sign, or choose another expert.
CLOSE_READ = {"bfloat16": 0.03, "float32": 0.005}
CLOSE_CHOICE = {"bfloat16": 0.005, "float32": 2e-6}


def firm_rows(dtype: str, cfg: dict, weights: dict, toks, margins: dict | None = None) -> np.ndarray:
    """Which positions' logits a run can be held to.  A delta head's output is divided by its root mean square, so where the
    read-out S^T q nearly cancels its direction hangs on the rounding of q and k; where the last chosen expert and the first
    that is not lie within a rounding of each other, either may be taken.  The row that follows is another row, and both
    are right.  margins: what `plain_gevipel.forward` has reported, where it has run already."""
    firm = np.ones(len(toks), dtype=bool)
    if margins is None:
        margins = plain_gevipel.new_margins()
        plain_gevipel.forward(cfg, weights, toks, margins=margins)
    for kind, limit in (("read", CLOSE_READ[dtype]), ("route", CLOSE_CHOICE[dtype])):
        for m in margins[kind]:
            firm &= m.numpy() >= limit
    return firm


def bound(dtype: str, cfg: dict, weights: dict, toks, exact: np.ndarray, firm=None) -> float:
    """What a row may differ by from the float64 plain implementation, measured on the request itself.  float32: three times
    what the plain implementation's worst firm row moves by when it runs in float32 or when what it keeps moves by a
    rounding's size at random, at least 2e-5.  bfloat16: three times what nine firm rows in ten stay below when it keeps
    its activations in bfloat16 (the rest holds rows where that run itself took another expert, or saw a row that did)."""
    firm = np.ones(len(toks), dtype=bool) if firm is None else firm
    size, runs = (2.0 ** -22, [{"dtype": torch.float32}]) if dtype == "float32" else (2.0 ** -9, [{"storage": torch.bfloat16}])
    runs.append({"noise": (size, 1)})
    errs = [row_errors(plain_gevipel.forward(cfg, weights, toks, **kw).numpy(), exact)[firm] for kw in runs]
    if dtype == "float32":
        return max(F32_TOL, 3.0 * max(float(e.max(initial=0.0)) for e in errs))
    return 3.0 * max(float(np.quantile(e, 0.9)) if e.size else 0.0 for e in errs)


def within(dtype: str, errors: np.ndarray, firm: np.ndarray, tol: float) -> bool:
    """float32: every firm row within the bound.  bfloat16: all but one firm row in twenty (and one more)."""
    over = int((np.asarray(errors)[firm] >= tol).sum())
    return over == 0 if dtype == "float32" else over <= 1 + 0.05 * int(firm.sum())


def load(folder):
    return plain_gevipel.load_folder(folder)
