"""The Korazen design without a GPU: configuration, the model as data, cache needs, the weight table, choices of kernel, and
the plain implementation against itself."""
import json
import math

import pytest
import torch

import plain_korazen
from korazen_models import CONFIGS, delta, dense, load, make_folder, model, random_config, sides, tokens

import longbow_quarrel_b200  # noqa: F401
from longbow_quarrel_b200 import architectures  # noqa: F401
from longbow_quarrel_b200.config import ConfigError, architecture_of
from longbow_quarrel_b200.config.korazen import KorazenConfig
from longbow_quarrel_b200.engine.model import Model
from longbow_quarrel_b200.kernels import attention as attention_kernels
from longbow_quarrel_b200.parts import make_part
from longbow_quarrel_b200.parts.base import KVNeed, Runtime, SeveralNeeds, StateNeed
from longbow_quarrel_b200.parts.spec import LayerSpec, PartSpec

CPU = torch.device("cpu")


def _model(data, dtype=torch.float32):
    arch = architecture_of(data)
    cfg = arch.config_from_dict(data)
    return cfg, arch.describe(cfg), Model(arch.describe(cfg), Runtime(CPU, dtype, 256))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_configuration_survives_the_round_trip(name):
    cfg = KorazenConfig.from_dict(CONFIGS[name])
    assert KorazenConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


def test_every_layer_has_one_cache_entry_with_what_its_mixer_keeps():
    cfg, spec, m = _model(CONFIGS["mixed"])
    assert [(e.layer, e.cache) for e in spec.schedule] == [(i, i) for i in range(5)]
    needs = m.cache_needs()
    assert needs[0] == SeveralNeeds((StateNeed((4, 32, 48), torch.float32), StateNeed((4, 2 * 2 * 32 + 4 * 48), torch.float32)))
    assert needs[1] == SeveralNeeds((KVNeed(1, 32, None, 64, chunk=64), StateNeed((2, 24, 40), torch.float32)))
    assert needs[3] == SeveralNeeds((KVNeed(2, 64, None, None, chunk=100), StateNeed((3, 32, 32), torch.float32)))
    assert needs[4].needs[1].shape == (2, 2 * 3 * 64 + 6 * 32)
    assert m.graph_safe


def test_the_weight_table_names_every_tensor_of_the_design():
    table = _model(CONFIGS["mixed"])[2].weight_table()
    assert table["embed"].shape == (200, 64) and table["embed.norm"].shape == (64,) and table["head"].shape == (200, 64)
    assert table["final.norm"].shape == (64,) and table["l0.norm1"].shape == table["l0.norm2"].shape == (64,)
    assert "l1.norm2" not in table and "l1.mlp.gate" not in table
    for n, shape in {"q": (64, 64), "k": (64, 64), "v": (192, 64), "q.conv": (64, 4), "k.conv": (64, 4), "v.conv": (192, 4), "b": (4, 64),
                     "A_log": (4,), "a1": (8, 64), "a2": (128, 8), "dt_bias": (128,), "g1": (12, 64), "g2": (192, 12), "norm": (48,),
                     "o": (64, 192)}.items():
        assert table["l0.mix." + n].shape == shape, n
    for n, shape in {"left.q": (128, 64), "left.q.b": (128,), "left.k": (32, 64), "left.k.b": (32,), "left.v": (64, 64), "left.v.b": (64,),
                     "left.q.norm": (32,), "left.k.norm": (32,), "left.g": (256, 64), "left.o": (64, 256), "left.o.b": (64,), "left.out": (64,),
                     "right.q": (48, 64), "right.k": (48, 64), "right.v": (80, 64), "right.g": (80, 64), "right.norm": (80,),
                     "right.o": (64, 80), "right.out": (64,)}.items():
        assert table["l1.mix." + n].shape == shape, n
    assert table["l0.mlp.gate"].shape == table["l0.mlp.up"].shape == (96, 64) and table["l0.mlp.down"].shape == (64, 96)
    assert len(table) == 4 + 3 * (15 + 1) + 2 * (21 - 2 + 1) + 3 * 4


def test_the_inner_sizes_may_come_from_the_tensors():
    data = json.loads(json.dumps(CONFIGS["only_delta"]))
    for key in ("rank", "gate_rank"):
        del data["layers"][0]["mixer"][key]
    table = _model(data)[2].weight_table()
    assert table["l0.mix.a1"].shape == (-1, 48) and table["l0.mix.a2"].shape == (64, -1)
    assert table["l0.mix.g1"].shape == (-1, 48) and table["l0.mix.g2"].shape == (96, -1)


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="delta"), "type"),
    (lambda c: c["layers"][0]["mixer"].update(heads=3, kv_heads=2), "multiple"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][1]["mixer"].pop("left"), "left"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(mask={"size": 0}), "size"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=34), "dims"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(decay=[0.5]), "decay"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("decay"), "decay"),
    (lambda c: c.update(logit_scale="2"), "logit_scale"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(change, message):
    data = json.loads(json.dumps(CONFIGS["mixed"]))
    change(data)
    with pytest.raises(ConfigError, match=message):
        KorazenConfig.from_dict(data)


def test_absent_keys_leave_their_mechanism_out():
    data = {"architecture": "Korazen", "vocab": 50, "width": 32, "norm": {"eps": 1e-5}, "layers": [
        {"type": "channel_delta", "mixer": {"heads": 2, "dim": 8, "conv": 4}},
        {"type": "parallel", "mlp": None, "mixer": {"left": {"heads": 2, "dim": 16}, "right": {"heads": 1, "dim": 8, "decay": [0.5]}}}]}
    cfg = KorazenConfig.from_dict(data)
    a, b = cfg.layers
    assert cfg.logit_scale == 1.0 and a.mlp is None and a.delta.kv_heads == 2 and a.delta.vdim == 8 and a.delta.rank is None
    assert b.left.block is None and b.left.rot_dims == 0 and b.left.scale == 0.25 and b.left.kv_heads == 2 and b.right.vdim == 8


def test_the_block_refuses_what_it_cannot_arrange():
    rt = Runtime(CPU, torch.float32, 64)
    norm = PartSpec("rms_norm", {"size": 8, "eps": 1e-5, "name": "norm1"})
    mixer = PartSpec("lightning", {"hidden_size": 8, "n_heads": 1, "key_dim": 4, "value_dim": 4, "decay": (0.5,), "eps": 1e-5})
    for parts in ({"mixer": mixer, "norm1": norm, "norm3": norm}, {"mixer": mixer, "norm1": norm, "norm2": norm},
                  {"mixer": mixer, "norm1": PartSpec("layer_norm", {"size": 8, "eps": 1e-5})}, {"mixer": mixer}):
        with pytest.raises(ValueError, match="post_norm|come together"):
            make_part("block", PartSpec("post_norm"), rt, layer=LayerSpec(prefix="l0.", arrangement="post_norm", parts=parts))
    with pytest.raises(ValueError, match="limit"):
        make_part("ffn", PartSpec("gated_mlp", {"hidden_size": 8, "intermediate_size": 8, "activation": "sigmoid_clamped"}), rt)
    with pytest.raises(ValueError, match="limit"):
        make_part("ffn", PartSpec("gated_mlp", {"hidden_size": 8, "intermediate_size": 8, "limit": 1.0}), rt)


def test_which_attention_kernel_takes_values_of_another_size():
    bf, f32 = torch.bfloat16, torch.float32
    kind = attention_kernels.prefill_kernel
    assert kind(bf, 128, vd=128) == kind(bf, 64) == "tc"
    assert kind(bf, 64, vd=128) == kind(bf, 128, vd=256) == kind(bf, 112, vd=224) == kind(bf, 48, vd=40) == "mma"
    assert kind(bf, 128, vd=264) is None and kind(bf, 128, vd=12) is None and kind(bf, 144, vd=64) is None and kind(f32, 64, vd=64) is None
    assert attention_kernels.decode_kernel(bf, 80, 160) and not attention_kernels.decode_kernel(bf, 96, 300)
    part = make_part("mixer", PartSpec("attention", {"hidden_size": 32, "n_heads": 4, "n_kv_heads": 2, "head_dim": 64, "scale": 0.1,
                                                     "value_dim": 128, "chunk": 70}), Runtime(CPU, bf, 64))
    assert set(part.step_needs()) == {"query_blocks64", attention_kernels.decode_work_name(4, 2, None, chunk=70)}


# ------------------------------------------------------------------ the plain implementation against itself

def test_plain_blocks_and_states_behave_as_the_design_says(tmp_path):
    """With the right side's output weight at zero only the blocks look back: a token outside a block changes nothing in
    it.  With it, and through the delta rule, the first token reaches the last."""
    folder = make_folder(tmp_path, "only_sides_wide_values", seed=1, std=0.3)
    cfg, weights = load(folder)
    base = tokens(60, cfg["vocab"], 2)
    odd = list(base)
    odd[23] = (odd[23] + 1) % cfg["vocab"]                  # the last position of the first block of 24
    alone = {**weights, "l0.mix.right.out": torch.zeros_like(weights["l0.mix.right.out"])}
    ref, out = plain_korazen.forward(cfg, alone, base), plain_korazen.forward(cfg, alone, odd)
    assert float((out[23] - ref[23]).abs().max()) > 1e-6
    assert float((out[24:] - ref[24:]).abs().max()) == 0.0 and float((out[:23] - ref[:23]).abs().max()) == 0.0
    odd = [(base[0] + 1) % cfg["vocab"]] + base[1:]
    assert float((plain_korazen.forward(cfg, weights, odd)[59] - plain_korazen.forward(cfg, weights, base)[59]).abs().max()) > 1e-9
    folder = make_folder(tmp_path, "only_delta", seed=1, std=0.3)
    cfg, weights = load(folder)
    assert float((plain_korazen.forward(cfg, weights, odd)[59] - plain_korazen.forward(cfg, weights, base)[59]).abs().max()) > 1e-9


def test_plain_mechanisms_one_by_one():
    torch.manual_seed(0)
    dt = torch.float64
    # the convolution is torch's grouped one with zeros ahead of the start, its last tap on the token itself
    z, w = torch.randn(9, 5, dtype=dt), torch.randn(5, 4, dtype=dt)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(z.T[None], (3, 0)), w[:, None, :], groups=5)[0].T
    assert torch.allclose(plain_korazen.causal_conv_silu(z, w), torch.nn.functional.silu(ref), atol=1e-12)
    assert torch.allclose(plain_korazen.softplus(z * 20), torch.nn.functional.softplus(z * 20), atol=1e-12)
    # a unit key written with b = 1 and nothing decayed is read back exactly, and writing it again replaces what it held
    k = plain_korazen.unit_length(torch.randn(1, 1, 6, dtype=dt))
    k = torch.cat([k, k])
    v = torch.randn(2, 1, 3, dtype=dt)
    ones = torch.ones(2, 1, dtype=dt)
    o = plain_korazen.delta_rule(k, k, v, ones, torch.ones(2, 1, 6, dtype=dt))
    assert torch.allclose(o, v, atol=1e-5)                   # the unit vectors' 1e-6 inside the root
    # b = 0 writes nothing; a decay of zero forgets everything
    assert float(plain_korazen.delta_rule(k, k, v, 0 * ones, torch.ones(2, 1, 6, dtype=dt)).abs().max()) == 0.0
    o = plain_korazen.delta_rule(k, k, v, torch.tensor([[1.0], [0.0]], dtype=dt), torch.zeros(2, 1, 6, dtype=dt))
    assert float(o[0].abs().max()) > 0 and float(o[1].abs().max()) == 0.0
    # halves with the clamp in force and far inside it
    w = {"gate": torch.eye(3, dtype=dt), "up": torch.eye(3, dtype=dt), "down": torch.eye(3, dtype=dt)}
    h = torch.tensor([[-9.0, 0.1, 9.0]], dtype=dt)
    got = plain_korazen.clamped_ffn(h, w, 2.0)[0]
    for x, y in zip(h[0].tolist(), got.tolist()):
        g, u = min(x, 2.0), max(-2.0, min(x, 2.0))
        assert math.isclose(y, g / (1 + math.exp(-1.702 * g)) * (u + 1), rel_tol=1e-12)


def test_a_configuration_drawn_at_random_runs_plain(tmp_path):
    import random
    for seed in (1, 2, 3):
        data = random_config(random.Random(seed))
        folder = make_folder(tmp_path, data, seed=seed)
        cfg, weights = load(folder)
        layers: list = []
        out = plain_korazen.forward(cfg, weights, tokens(20, cfg["vocab"], seed), layers_out=layers)
        assert out.shape == (20, cfg["vocab"]) and torch.isfinite(out).all() and len(layers) == len(cfg["layers"])


def test_a_layer_is_built_from_any_sizes():
    data = model(24, 30, [delta(6, 3, 4, 3, conv=3, rank=1, gate_rank=5, mlp=dense(8, 0.1)), sides((2, 1, 6, 10, 0.5, 3, (2, 10.0)), (3, 5, (0.5,)))])
    table = _model(data)[2].weight_table()
    assert table["l0.mix.g2"].shape == (18, 5) and table["l1.mix.left.g"].shape == (20, 24) and table["l0.mlp.up"].shape == (8, 24)
