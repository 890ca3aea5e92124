"""The Gevipel design without a GPU: configuration, the model as data, cache needs, the weight table, what parts refuse, and
the plain implementation against itself."""
import json
import math

import pytest
import torch

import plain_gevipel
from gevipel_models import CONFIGS, attn, delta, latent, load, make_folder, model, moe, random_config, rewrite, tokens

import longbow_quarrel_b200  # noqa: F401
from longbow_quarrel_b200 import architectures  # noqa: F401
from longbow_quarrel_b200.config import ConfigError, architecture_of
from longbow_quarrel_b200.config.gevipel import GevipelConfig
from longbow_quarrel_b200.engine.model import Model
from longbow_quarrel_b200.parts import make_part
from longbow_quarrel_b200.parts.base import KVNeed, Runtime, SeveralNeeds, StateNeed
from longbow_quarrel_b200.parts.rope import pair_order
from longbow_quarrel_b200.parts.spec import LayerSpec, PartSpec

CPU = torch.device("cpu")


def _model(data, dtype=torch.float32):
    arch = architecture_of(data)
    cfg = arch.config_from_dict(data)
    return cfg, arch.describe(cfg), Model(arch.describe(cfg), Runtime(CPU, dtype, 256))


@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_a_configuration_survives_the_round_trip(name):
    cfg = GevipelConfig.from_dict(CONFIGS[name])
    assert GevipelConfig.from_dict(json.loads(json.dumps(cfg.to_dict()))) == cfg


def test_every_run_of_a_layer_has_a_cache_entry_of_its_own():
    cfg, spec, m = _model(CONFIGS["mixed"])
    # the embedding's output joins ahead of the second pass only, as a layer that keeps nothing
    assert [e.layer for e in spec.schedule] == [0, 1, 2, 3, 5, 1, 2, 3, 4]
    assert [e.cache for e in spec.schedule] == list(range(9))
    needs = m.cache_needs()
    assert needs[0] == KVNeed(1, 40 + 8, None, values=False)
    assert needs[1] == needs[5] == SeveralNeeds((StateNeed((4, 32, 48), torch.float32), StateNeed((4, 2 * 2 * 32 + 4 * 48), torch.float32)))
    assert needs[2] == needs[6] == KVNeed(2, 32, 64)
    assert needs[4] is None and needs[8] == KVNeed(1, 64, 100)
    assert m.graph_safe
    # one pass: nothing joins
    cfg, spec, m = _model(CONFIGS["only_loop_once"])
    assert [e.layer for e in spec.schedule] == [0, 1, 2] and len(spec.layers) == 3
    assert not m._keeps_embedding


def test_the_weight_table_names_every_tensor_of_the_design():
    table = _model(CONFIGS["mixed"])[2].weight_table()
    assert table["embed"].shape == table["head"].shape == (200, 64)
    assert table["final.norm"].shape == table["final.norm.b"].shape == (64,)
    for n in ("norm1", "norm1b", "norm2", "norm2b"):
        assert table[f"l0.{n}"].shape == table[f"l0.{n}.b"].shape == (64,)
    assert "l3.norm2" not in table and "l3.norm2b" not in table and "l3.mlp.router" not in table
    for n, shape in {"q": (128, 64), "dkv": (48, 64), "dkv.norm": (40,), "uk": (96, 40), "uv": (128, 40), "sink": (4,), "o": (64, 128)}.items():
        assert table["l0.mix." + n].shape == shape, n
    for n, shape in {"q": (64, 64), "k": (64, 64), "v": (192, 64), "q.conv": (64, 4), "k.conv": (64, 4), "v.conv": (192, 4), "b": (4, 64),
                     "a": (4, 64), "A_log": (4,), "dt_bias": (4,), "g": (192, 64), "norm": (48,), "o": (64, 192)}.items():
        assert table["l1.mix." + n].shape == shape, n
    for n, shape in {"q": (128, 64), "k": (64, 64), "q.norm": (32,), "k.norm": (32,), "o": (64, 128)}.items():
        assert table["l2.mix." + n].shape == shape, n
    assert table["l1.mlp.router"].shape == (5, 64) and table["l1.mlp.correction"].shape == (5,)
    assert table["l1.mlp.e4.up"].shape == (24, 64) and table["l1.mlp.e4.down"].shape == (64, 24) and "l1.mlp.e5.up" not in table
    assert len(table) == 4 + (8 + 7) + (8 + 13) + (8 + 5) + (4 + 13) + (8 + 5) + sum(2 + 2 * e for e in (6, 5, 6, 4))


@pytest.mark.parametrize("change, message", [
    (lambda c: c["layers"][0].update(type="mamba"), "type"),
    (lambda c: c["layers"][1]["mixer"].update(heads=3, kv_heads=2), "multiple"),
    (lambda c: c["layers"][1]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][1]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][1]["mixer"].pop("dim"), "dim"),
    (lambda c: c["layers"][2]["mixer"].update(vdim=16), "vdim"),
    (lambda c: c["layers"][2]["mixer"].update(mask={"size": 0}), "size"),
    (lambda c: c["layers"][2]["mixer"].update(q_temp={"coef": 0.1}), "every"),
    (lambda c: c["layers"][2]["mixer"].update(q_temp={"coef": 0.1, "every": 0}), "every"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=10), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].pop("base"), "base"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "top"),
    (lambda c: c["layers"][0]["mlp"].pop("expert"), "expert"),
    (lambda c: c["loop"].update(stop=6), "loop"),
    (lambda c: c["loop"].update(times=0), "times"),
    (lambda c: c["embedding"].update(scale="2"), "scale"),
    (lambda c: c.update(residual_mult="x"), "residual_mult"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_configuration_errors_name_the_key(change, message):
    data = json.loads(json.dumps(CONFIGS["mixed"]))
    change(data)
    with pytest.raises(ConfigError, match=message):
        GevipelConfig.from_dict(data)


def test_absent_keys_leave_their_mechanism_out():
    data = {"architecture": "Gevipel", "vocab": 50, "width": 32, "norm": {"eps": 1e-5}, "layers": [
        {"type": "delta", "mixer": {"heads": 2, "dim": 8, "conv": 4}},
        {"type": "attention", "mixer": {"heads": 2, "dim": 16}},
        {"type": "latent_attention", "mlp": None, "mixer": {"heads": 2, "dim": 12, "rot_dim": 4, "kv_rank": 8}}]}
    cfg = GevipelConfig.from_dict(data)
    a, b, c = (layer.mixer for layer in cfg.layers)
    assert cfg.embedding_scale == cfg.residual_mult == 1.0 and cfg.loop is None and all(layer.mlp is None for layer in cfg.layers)
    assert a.kv_heads == 2 and a.vdim == 8 and b.window is None and b.temp_coef is None and b.scale == 0.25
    assert c.rot_dims is None and c.vdim == 12 and c.scale == 0.25
    assert b.slopes == (2.0 ** -4, 2.0 ** -8)
    assert len(_model(data)[1].schedule) == 3


def test_parts_refuse_what_they_cannot_do():
    rt = Runtime(CPU, torch.float32, 64)
    base = {"hidden_size": 8, "n_heads": 2, "n_kv_heads": 2, "head_dim": 4, "scale": 1.0}
    for more, message in (({"values": "keys", "value_dim": 6}, "keys' size"), ({"values": "queries"}, "values"),
                          ({"values": "keys", "own_kv": False}, "keys of their own"), ({"distance_slopes": (0.5,)}, "slopes")):
        with pytest.raises(ValueError, match=message):
            make_part("mixer", PartSpec("attention", {**base, **more}), rt)
    with pytest.raises(ValueError, match="value size"):
        make_part("mixer", PartSpec("head_delta", {"hidden_size": 8, "n_heads": 1, "key_dim": 4, "value_dim": 257, "taps": 4, "eps": 1e-5}), rt)
    with pytest.raises(ValueError, match="not both"):
        make_part("embedding", PartSpec("token_embedding", {"vocab_size": 8, "hidden_size": 8, "name": "e", "scale": 2.0,
                                                            "norm": PartSpec("rms_norm", {"size": 8, "eps": 1e-5})}), rt)
    with pytest.raises(ValueError, match="no places"):
        make_part("block", PartSpec("stream_add"), rt, layer=LayerSpec(prefix="l.", arrangement="stream_add", parts={"norm1": None}))


def test_which_sandwich_takes_the_kernel_for_norms_of_any_kind():
    rt = Runtime(CPU, torch.float32, 64)
    mixer = PartSpec("attention", {"hidden_size": 8, "n_heads": 1, "n_kv_heads": 1, "head_dim": 4, "scale": 1.0})

    def block(kind, **params):
        norms = {n: PartSpec(kind, {"size": 8, "eps": 1e-5, "name": n}) for n in ("norm1", "norm1b")}
        return make_part("block", PartSpec("sandwich_norm", params), rt, layer=LayerSpec(prefix="l.", arrangement="sandwich_norm",
                                                                                          parts={"mixer": mixer, **norms}))
    plain, scaled, layered = block("rms_norm"), block("rms_norm", residual_scale=0.5), block("layer_norm")
    assert not plain.general and scaled.general and layered.general
    for b in (plain, scaled, layered):
        b.load({n: torch.ones(s.shape) for n, s in b.weights().items()})
    assert plain.input_norm(4)[1] == 1e-5 and scaled.input_norm(4) is not None and layered.input_norm(4) is None
    gain, bias, eps, center = layered.first_norm()
    assert gain.shape == bias.shape == (8,) and eps == 1e-5 and center
    assert scaled.first_norm()[1] is None and not scaled.first_norm()[3]


def test_interleaved_pairs_of_the_latent_layer_are_reordered_once_at_load():
    data = model(24, 30, [latent(2, 6, 8, 10, 12)])
    m = _model(data)[2]
    g = torch.Generator().manual_seed(0)
    weights = {n: torch.randn(s.shape, generator=g) for n, s in m.weight_table().items()}
    m.load(weights)
    part, order = m.blocks[0].mixer, pair_order(8, 8)
    q = weights["l0.mix.q"].reshape(2, 14, 24)
    assert torch.equal(part.w_uq.tensor.reshape(2, 14, 24)[:, :6], q[:, :6])
    assert torch.equal(part.w_uq.tensor.reshape(2, 14, 24)[:, 6:], q[:, 6:][:, order])
    assert torch.equal(part.w_down.tensor[:12], weights["l0.mix.dkv"][:12])
    assert torch.equal(part.w_down.tensor[12:], weights["l0.mix.dkv"][12:][order])
    assert torch.equal(part.sinks, weights["l0.mix.sink"])


# ------------------------------------------------------------------ the plain implementation against itself

def test_plain_windows_and_states_behave_as_the_design_says(tmp_path):
    """A token outside a window changes nothing inside it; through the delta rule and the latent rows the first token reaches
    the last."""
    folder = make_folder(tmp_path, "only_attention_mma", seed=1, std=0.3)
    cfg, weights = load(folder)
    base = tokens(60, cfg["vocab"], 2)
    odd = list(base)
    odd[23] = (odd[23] + 1) % cfg["vocab"]
    ref, out = plain_gevipel.forward(cfg, weights, base), plain_gevipel.forward(cfg, weights, odd)
    assert float((out[42] - ref[42]).abs().max()) > 1e-9                     # the window of 20 ends here
    assert float((out[43:] - ref[43:]).abs().max()) == 0.0 and float((out[:23] - ref[:23]).abs().max()) == 0.0
    for name in ("only_delta", "only_latent"):
        folder = make_folder(tmp_path, name, seed=1, std=0.2)
        cfg, weights = load(folder)
        base = tokens(60, cfg["vocab"], 2)
        odd = [(base[0] + 1) % cfg["vocab"]] + base[1:]
        assert float((plain_gevipel.forward(cfg, weights, odd)[59] - plain_gevipel.forward(cfg, weights, base)[59]).abs().max()) > 1e-9


def test_plain_loop_takes_the_embedding_in_ahead_of_every_pass_but_the_first(tmp_path):
    """With every branch's norm at zero the layers add nothing: the stream is the scaled embedding times the number of passes."""
    folder = make_folder(tmp_path, "only_loop", seed=1)

    def change(w):
        for n in w:
            if "norm1b" in n or "norm2b" in n:
                w[n].zero_()
    rewrite(folder, change)
    cfg, weights = load(folder)
    layers: list = []
    plain_gevipel.forward(cfg, weights, [3, 4], layers_out=layers)
    e = weights["embed"][[3, 4]].double() * cfg["embedding"]["scale"]
    for i, x in enumerate(layers):
        assert torch.allclose(x, e * (1 + i // 2), atol=1e-12)
    assert len(layers) == 6


def test_plain_mechanisms_one_by_one():
    torch.manual_seed(0)
    dt = torch.float64
    x, g, b = torch.randn(3, 7, dtype=dt) + 2, torch.randn(7, dtype=dt), torch.randn(7, dtype=dt)
    assert torch.allclose(plain_gevipel.layer_norm(x, g, b, 1e-5), torch.nn.functional.layer_norm(x, (7,), g, b, 1e-5), atol=1e-12)
    # the convolution is torch's grouped one with zeros ahead of the start, its last tap on the token itself
    z, w = torch.randn(9, 5, dtype=dt), torch.randn(5, 4, dtype=dt)
    ref = torch.nn.functional.conv1d(torch.nn.functional.pad(z.T[None], (3, 0)), w[:, None, :], groups=5)[0].T
    assert torch.allclose(plain_gevipel.causal_conv_silu(z, w), torch.nn.functional.silu(ref), atol=1e-12)
    # a unit key written with b = 1 and nothing decayed is read back; writing it again replaces what it held; a decay of zero forgets
    k = plain_gevipel.unit_length(torch.randn(1, 1, 6, dtype=dt))
    k, v, ones = torch.cat([k, k]), torch.randn(2, 1, 3, dtype=dt), torch.ones(2, 1, dtype=dt)
    assert torch.allclose(plain_gevipel.delta_rule(k, k, v, ones, ones), v, atol=1e-5)
    assert float(plain_gevipel.delta_rule(k, k, v, 0 * ones, ones).abs().max()) == 0.0
    o = plain_gevipel.delta_rule(k, k, v, torch.tensor([[1.0], [0.0]], dtype=dt), 0 * ones)
    assert float(o[0].abs().max()) > 0 and float(o[1].abs().max()) == 0.0
    # pairs of neighbours turn; at position 0 nothing does; lengths stay
    x = torch.randn(4, 2, 6, dtype=dt)
    y = plain_gevipel.rotate_neighbours(x, {"dims": 4, "base": 10.0})
    assert torch.equal(y[0], x[0]) and torch.equal(y[:, :, 4:], x[:, :, 4:])
    assert torch.allclose(y[..., :2].norm(dim=-1), x[..., :2].norm(dim=-1)) and not torch.allclose(y[3, :, :2], x[3, :, :2])
    u, w2 = complex(x[3, 0, 2], x[3, 0, 3]), complex(y[3, 0, 2], y[3, 0, 3])
    a = 3 * 10.0 ** (-2.0 / 4)
    assert abs(u * complex(math.cos(a), math.sin(a)) - w2) < 1e-12
    # one more term without a key; slopes; the temperature's steps
    s = torch.randn(2, 5, dtype=dt)
    p = plain_gevipel.softmax_rows(s, torch.tensor([0.3, -50.0], dtype=dt))
    assert torch.allclose(p[0], torch.softmax(torch.cat([s[0], torch.tensor([0.3], dtype=dt)]), 0)[:-1]) and math.isclose(float(p[1].sum()), 1.0)
    assert plain_gevipel.slopes(8).tolist() == [2.0 ** -(h + 1) for h in range(8)]
    t = plain_gevipel.temperature(9, {"q_temp": {"coef": 0.5, "every": 4}})
    assert t[:3].tolist() == [1.0] * 3 and math.isclose(t[3], 1 + 0.5 * math.log(2)) and math.isclose(t[7], 1 + 0.5 * math.log(3))
    # the correction chooses, the plain scores weigh
    z, c = torch.tensor([0.0, 1.0, 2.0], dtype=dt), torch.tensor([5.0, 0.0, 0.0], dtype=dt)
    experts, weights, gap = plain_gevipel.route(z, c, 2)
    assert experts == [0, 2] and torch.allclose(weights, torch.softmax(z, 0)[[0, 2]]) and gap > 0


def test_a_configuration_drawn_at_random_runs_plain(tmp_path):
    import random
    for seed in (1, 2, 3):
        data = random_config(random.Random(seed))
        folder = make_folder(tmp_path, data, seed=seed)
        cfg, weights = load(folder)
        layers: list = []
        out = plain_gevipel.forward(cfg, weights, tokens(20, cfg["vocab"], seed), layers_out=layers)
        assert out.shape == (20, cfg["vocab"]) and torch.isfinite(out).all() and len(layers) == len(plain_gevipel.layer_order(cfg))


def test_a_layer_is_built_from_any_sizes():
    data = model(24, 30, [delta(6, 3, 4, 3, conv=3, mlp=moe(2, 1, 5)), attn(4, 1, 6, window=3), latent(3, 5, 2, 7, 9)])
    table = _model(data)[2].weight_table()
    assert table["l0.mix.g"].shape == (18, 24) and table["l1.mix.k"].shape == (6, 24) and table["l2.mix.uv"].shape == (21, 9)
