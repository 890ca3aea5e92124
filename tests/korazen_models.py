"""Small Korazen configurations and model folders with random weights, for the tests of this design.

The configurations differ from each other in every size and option: delta-rule heads of 8 to 200 key channels and 5 to 72
values, as many key heads as value heads and fewer, convolutions of 1, 2, 3, 4, 5 and 7 taps, inner sizes of 1 to 24 that
differ between decays and gate; attention in blocks of 1, 7, 24, 64, 70 and 100 positions and over all of them, with values
wider and narrower than keys, rotation of all, a part and none of a head, several scales; fixed-decay heads of 8 to 80 key
channels with decays of 0.2 to 1; feed-forwards with limits of 0.3 to 7 behind either mixer, and layers without one; logit
scales of 0.5 to 3; widths and head sizes that are no multiples of 8.
"""
from __future__ import annotations

import json
from pathlib import Path

import numpy as np
import torch

import plain_korazen


def delta(heads, kv_heads, dim, vdim, conv=4, rank=8, gate_rank=None, mlp=None):
    return {"type": "channel_delta", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rank": rank,
                      "gate_rank": rank if gate_rank is None else gate_rank}}


def sides(left, right, mlp=None):
    """left: (heads, kv_heads, dim, vdim, scale | None, block | None, (dims, base) | None); right: (dim, vdim, decays)."""
    h, g, dim, vdim, scale, block, rot = left
    lm = {"heads": h, "kv_heads": g, "dim": dim, "vdim": vdim, "scale": dim ** -0.5 if scale is None else scale}
    if block is not None:
        lm["mask"] = {"size": block}
    if rot is not None:
        lm["rot"] = {"dims": rot[0], "base": rot[1]}
    rdim, rvdim, decay = right
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": lm, "right": {"heads": len(decay), "dim": rdim, "vdim": rvdim, "decay": list(decay)}}}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def model(width, vocab, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Korazen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


CONFIGS = {
    # one mechanism each
    "only_delta": model(48, 120, [delta(4, 2, 16, 24, conv=4, rank=5, gate_rank=7)], logit_scale=1.5),
    "only_delta_even": model(64, 90, [delta(2, 2, 64, 64, conv=3, rank=16)]),
    "only_delta_wide_keys": model(40, 100, [delta(2, 1, 200, 20, conv=5, rank=1, gate_rank=3)], eps=1e-6),
    "only_delta_odd": model(36, 77, [delta(3, 3, 20, 37, conv=7, rank=24, gate_rank=2)], logit_scale=0.5),
    "only_delta_no_past": model(32, 80, [delta(6, 2, 8, 5, conv=1, rank=3)]),
    "only_delta_two_taps": model(56, 80, [delta(1, 1, 96, 72, conv=2, rank=8, mlp=dense(40, 0.5))]),
    "only_sides": model(64, 140, [sides((2, 1, 64, 64, None, 40, (64, 3e4)), (32, 48, (0.9, 1.0)), mlp=dense(40, 1.2))], logit_scale=3.0),
    "only_sides_wide_values": model(48, 110, [sides((4, 2, 16, 32, 0.3, 24, (16, 100.0)), (24, 8, (0.5, 0.99, 0.2)))]),
    "only_sides_narrow_values": model(64, 110, [sides((2, 2, 128, 40, 0.08, 70, (32, 1e4)), (8, 72, (0.97,)))]),
    "only_sides_very_wide_values": model(64, 90, [sides((3, 1, 48, 160, None, 100, (8, 500.0)), (80, 40, (0.8, 0.999)))]),
    "only_sides_open": model(36, 100, [sides((3, 3, 26, 42, 0.25, None, None), (20, 12, (0.7, 0.95)), mlp=dense(36, 7.0))], eps=1e-6),
    # whole models
    "mixed": model(64, 200, [
        delta(4, 2, 32, 48, conv=4, rank=8, gate_rank=12, mlp=dense(96, 1.5)),
        sides((4, 1, 32, 64, 0.2, 64, (16, 1e4)), (24, 40, (0.6, 0.99)), mlp=None),
        delta(2, 2, 24, 16, conv=3, rank=4, mlp=None),
        sides((2, 2, 64, 64, None, 100, (64, 5e4)), (32, 32, (0.9, 0.3, 0.999)), mlp=dense(72, 0.8)),
        delta(6, 3, 64, 32, conv=2, rank=16, gate_rank=9, mlp=dense(64, 3.0))], logit_scale=1.25),
    "odd": model(44, 131, [
        sides((3, 1, 20, 12, None, 7, (4, 50.0)), (36, 20, (0.85, 0.5)), mlp=dense(50, 0.3)),
        delta(3, 1, 36, 28, conv=5, rank=3, gate_rank=1, mlp=None),
        sides((5, 5, 12, 20, 0.4, 1, None), (12, 28, (0.9,)), mlp=None),
        delta(2, 2, 12, 44, conv=1, rank=2, mlp=dense(36, 2.0))], eps=1e-6, logit_scale=2.5),
    "wide": model(128, 300, [
        delta(4, 4, 128, 64, conv=4, rank=32, mlp=None),
        sides((4, 2, 128, 128, None, 100, (128, 1e4)), (64, 64, (0.9, 0.99)), mlp=dense(160, 1.0)),
        sides((4, 1, 64, 128, 0.1, 64, (32, 1e3)), (64, 32, (0.7, 0.95, 0.999)), mlp=None),
        delta(2, 1, 64, 128, conv=4, rank=16, gate_rank=24, mlp=dense(128, 2.0))], logit_scale=0.7),
}


def random_config(rng) -> dict:
    """A configuration whose sizes and options nobody chose."""
    layers = []
    for _ in range(rng.randint(2, 5)):
        mlp = dense(rng.choice([24, 40, 64]), rng.choice([0.4, 1.0, 2.5])) if rng.random() < 0.5 else None
        g = rng.randint(1, 3)
        h = g * rng.randint(1, 3)
        if rng.random() < 0.5:
            layers.append(delta(h, g, rng.choice([8, 16, 40, 64]), rng.choice([8, 12, 33, 48]), conv=rng.randint(1, 6),
                                rank=rng.randint(1, 12), gate_rank=rng.randint(1, 12), mlp=mlp))
        else:
            dim = rng.choice([8, 16, 32, 64])
            rot = (rng.choice([d for d in (2, 4, 8, dim) if d <= dim]), rng.choice([100.0, 1e4])) if rng.random() < 0.8 else None
            decay = [rng.choice([0.3, 0.9, 0.99, 0.999]) for _ in range(rng.randint(1, 3))]
            layers.append(sides((h, g, dim, rng.choice([dim, 2 * dim, 24]), rng.choice([None, 0.1, 0.25]), rng.choice([None, 3, 17, 64, 90]), rot),
                                (rng.choice([8, 24, 40]), rng.choice([8, 24, 48]), decay), mlp=mlp))
    return model(rng.choice([24, 40, 56, 64, 72]), rng.choice([77, 128, 200]), layers, eps=rng.choice([1e-5, 1e-6]),
                 logit_scale=rng.choice([0.5, 1.0, 2.2]))


def make_folder(tmp, name, seed: int = 0, std: float = 0.1, gain_std: float = 0.2, dtype=torch.bfloat16, keep_ranks: bool = True) -> Path:
    """A model folder with random weights, written by the framework's random-weights mode.  keep_ranks False: config.json
    does not say the inner sizes of the decays' and the gate's products (they are then read from the tensors' shapes)."""
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
    folder = write_random_model(Path(tmp) / f"korazen_{label}_{seed}", cfg.to_dict(), table, seed, dtype, std, gain_std)
    if not keep_ranks:
        data = json.loads((folder / "config.json").read_text())
        for layer in data["layers"]:
            for key in ("rank", "gate_rank"):
                layer["mixer"].pop(key, None)
        (folder / "config.json").write_text(json.dumps(data, indent=2))
    return folder


def rewrite(folder, change) -> None:
    """Change a folder's weights in place: change(weights) edits the dictionary of tensors."""
    from longbow_quarrel_b200.weights import write_safetensors
    weights = plain_korazen.read_safetensors(Path(folder) / "model.safetensors")
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


# Of what a read-out would be if nothing in it cancelled: rounding to bfloat16 may turn its sign; (float32) rounding's
# errors are blown up hundreds of times.
CLOSE_CALL = {"bfloat16": 0.03, "float32": 0.005}


def firm_rows(dtype: str, cfg: dict, weights: dict, toks, margins: list | None = None) -> np.ndarray:
    """Which positions' logits a run can be held to.  A head's output is divided by its root mean square, so where
    the read-out S^T q nearly cancels (at a sequence's first position it is a multiple of q . k alone) its direction
    hangs on the rounding of q and k, and the row that follows is another row; both are right.  Such positions are left out, and in
    bfloat16 the eight after them as well, for which the other row is much of what they see.
    margins: what `plain_korazen.forward` has reported, where it has run already."""
    firm = np.ones(len(toks), dtype=bool)
    if margins is None:
        margins = []
        plain_korazen.forward(cfg, weights, toks, margins=margins)
    for m in margins:
        for p in np.nonzero(m.numpy() < CLOSE_CALL[dtype])[0]:
            firm[p:p + (1 if dtype == "float32" else 9)] = False
    return firm


def bound(dtype: str, cfg: dict, weights: dict, toks, exact: np.ndarray, firm=None) -> float:
    """What a row may differ by from the float64 plain implementation, measured on the request itself: three times
    what the plain implementation moves by when it runs in float32 (at least 2e-5), or when it keeps its
    activations in bfloat16, or when what it keeps moves by a rounding's size at random.  The request's worst (firm) row."""
    firm = np.ones(len(toks), dtype=bool) if firm is None else firm
    size, runs = (2.0 ** -22, [{"dtype": torch.float32}]) if dtype == "float32" else (2.0 ** -9, [{"storage": torch.bfloat16}])
    runs.append({"noise": (size, 1)})
    worst = max(float(row_errors(plain_korazen.forward(cfg, weights, toks, **kw).numpy(), exact)[firm].max(initial=0.0)) for kw in runs)
    return max(F32_TOL if dtype == "float32" else 0.0, 3.0 * worst)


def load(folder):
    return plain_korazen.load_folder(folder)
