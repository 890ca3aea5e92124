"""The Korazen decoder, described from parts.

A list of layers that norm what a sublayer returns and nothing else: the sublayers read the residual stream as it is
(`post_norm`), and the embedding's rows are normed once, ahead of the first layer.  A layer's mixer is "channel_delta"
(the gated delta rule with a decay per key channel behind short convolutions) or "parallel" (softmax attention inside
blocks of positions, with biases, weighted unit norms of q and k per head, rotation of a head's first dimensions and a
sigmoid gate per value, side by side with linear attention of fixed decays; each side's output is normed over the
width with a weight of its own, and the layer takes half the sum).  The feed-forward is gated with clamped halves.  The
head has its own matrix; the logits are multiplied by a constant.

Tensor names: `embed`, `embed.norm`, `l<i>.norm1 | norm2`, `l<i>.mix.<q|k|v>` with `.conv`, `l<i>.mix.<b|A_log|a1|a2|dt_bias|
g1|g2|norm|o>`, or `l<i>.mix.left.<q|k|v|o>` with `.b`, `l<i>.mix.left.<q.norm|k.norm|g|out>` and
`l<i>.mix.right.<q|k|v|g|o|norm|out>`; `l<i>.mlp.<gate|up|down>`; `final.norm`, `head`.
"""
from __future__ import annotations

from ..config.korazen import KorazenConfig, KorazenLayer
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _norm(cfg: KorazenConfig, name: str, **more) -> PartSpec:
    return PartSpec("rms_norm", {"size": cfg.width, "eps": cfg.norm_eps, "name": name, **more})


def _mixer(cfg: KorazenConfig, layer: KorazenLayer) -> PartSpec:
    if layer.type == "channel_delta":
        d = layer.delta
        names = ("q", "k", "v", "b", "A_log", "a1", "a2", "dt_bias", "g1", "g2", "norm", "o")
        return PartSpec("channel_delta", {"hidden_size": cfg.width, "n_heads": d.heads, "n_kv_heads": d.kv_heads, "key_dim": d.dim,
                                          "value_dim": d.vdim, "taps": d.conv, "eps": cfg.norm_eps, "rank": d.rank,
                                          "gate_rank": d.gate_rank, "names": {n: f"mix.{n}" for n in names}})
    a, r = layer.left, layer.right
    names = {n: n for n in ("q", "k", "v", "o", "g")}
    names.update({f"{n}_bias": f"{n}.b" for n in ("q", "k", "v", "o")}, q_norm="q.norm", k_norm="k.norm")
    left = {"hidden_size": cfg.width, "n_heads": a.heads, "n_kv_heads": a.kv_heads, "head_dim": a.dim, "value_dim": a.vdim,
            "scale": a.scale, "chunk": a.block, "bias": True, "out_bias": True, "qk_norm": "head_gain", "norm_eps": cfg.norm_eps,
            "gate": "sigmoid", "names": names}
    if a.rot_dims:
        left["position"] = PartSpec("rope", {"head_dim": a.dim, "theta": a.rot_base, "rotary_dims": a.rot_dims})
    right = {"hidden_size": cfg.width, "n_heads": r.heads, "key_dim": r.dim, "value_dim": r.vdim, "decay": r.decay, "eps": cfg.norm_eps}
    return PartSpec("side_by_side", {"left": PartSpec("attention", left), "right": PartSpec("lightning", right),
                                     "left_scale": 0.5, "right_scale": 0.5, "left_prefix": "mix.left.", "right_prefix": "mix.right.",
                                     "out_norms": {"size": cfg.width, "eps": cfg.norm_eps, "left": "mix.left.out", "right": "mix.right.out"}})


def describe(cfg: KorazenConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        parts = dict(mixer=_mixer(cfg, layer), norm1=_norm(cfg, "norm1"))
        if layer.mlp is not None:
            ffn = {"hidden_size": cfg.width, "intermediate_size": layer.mlp.ff, "activation": "sigmoid_clamped", "limit": layer.mlp.limit,
                   "names": {n: f"mlp.{n}" for n in ("gate", "up", "down")}}
            parts.update(ffn=PartSpec("gated_mlp", ffn), norm2=_norm(cfg, "norm2"))
        layers.append(LayerSpec(prefix=f"l{i}.", arrangement="post_norm", parts=parts))
    return ModelSpec(
        name="Korazen", hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed",
                                               "norm": _norm(cfg, "embed.norm")}),
        layers=tuple(layers), schedule=tuple(ScheduleEntry(layer=i, cache=i) for i in range(len(layers))),
        # The logits' factor rides in the final norm's gain: W (g x) c = W (c g x), the product c g made once in 32-bit.
        final_norm=_norm(cfg, "final.norm", multiplier=cfg.logit_scale),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "head"}),
        max_positions=cfg.max_positions)


register_architecture("Korazen", KorazenConfig.from_dict, describe)
