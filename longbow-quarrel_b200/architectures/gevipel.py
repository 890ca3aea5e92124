"""The Gevipel decoder, described from parts.

A list of layers that norm every branch on both sides with layer norms (weight and bias) and multiply it by a constant as it
joins the stream, each with its own mixer and sizes: "delta" (the gated delta rule with one decay per head behind short
convolutions), "attention" (grouped softmax attention without rotation whose values are the keys as projected: weighted unit
norms of q and k per head, a query temperature that grows with the position, a sliding window, scores that fall with the
distance at a rate of each head's own) or "latent_attention" (keys and values as per-head maps of one normed latent row per
token plus one rotated key part shared by all heads, a learned term in the softmax denominator).  The feed-forward is routed
experts with the square of relu (softmax router; the choice is made by the scores plus a correction, the weights are the
chosen scores as they are), or absent.  The embedding's rows are multiplied by a constant; a stretch of layers may run several
times with the same weights, each pass but the first starts with x <- x + e, e the embedding's output, and every run of a
layer has its own cache entry.  The head has its own matrix.

Tensor names: `embed`, `l<i>.norm1 | norm1b | norm2 | norm2b` with biases `<name>.b`, `l<i>.mix.<q|k|v>` with `.conv`,
`l<i>.mix.<b|a|A_log|dt_bias|norm|g|o>`, or `l<i>.mix.<q|k|o|q.norm|k.norm>`, or `l<i>.mix.<q|dkv|dkv.norm|uk|uv|sink|o>`;
`l<i>.mlp.router`, `l<i>.mlp.correction`, `l<i>.mlp.e<j>.<up|down>`; `final.norm`, `final.norm.b`, `head`.
"""
from __future__ import annotations

from ..config.gevipel import GevipelConfig, GevipelLayer
from ..config.registry import register_architecture
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry


def _norm(cfg: GevipelConfig, name: str) -> PartSpec:
    return PartSpec("layer_norm", {"size": cfg.width, "eps": cfg.norm_eps, "name": name})


def _mixer(cfg: GevipelConfig, layer: GevipelLayer) -> PartSpec:
    m = layer.mixer
    if layer.type == "delta":
        names = ("q", "k", "v", "b", "a", "A_log", "dt_bias", "norm", "g", "o")
        return PartSpec("head_delta", {"hidden_size": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "key_dim": m.dim,
                                       "value_dim": m.vdim, "taps": m.conv, "eps": cfg.norm_eps,
                                       "names": {n: "mix." + n for n in names}})
    if layer.type == "attention":
        return PartSpec("attention", {"hidden_size": cfg.width, "n_heads": m.heads, "n_kv_heads": m.kv_heads, "head_dim": m.dim,
                                      "scale": m.scale, "window": m.window, "values": "keys", "qk_norm": "head_gain",
                                      "norm_eps": cfg.norm_eps, "distance_slopes": m.slopes,
                                      "q_temp": (m.temp_coef, m.temp_every) if m.temp_coef is not None else None,
                                      "names": {"q": "mix.q", "k": "mix.k", "o": "mix.o", "q_norm": "mix.q.norm", "k_norm": "mix.k.norm"}})
    position = None
    if m.rot_dims is not None:
        position = PartSpec("rope", {"head_dim": m.rot_dim, "theta": m.rot_base, "rotary_dims": m.rot_dims, "layout": "interleaved"})
    return PartSpec("latent_attention", {
        "hidden_size": cfg.width, "n_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "q_rank": None,
        "kv_rank": m.kv_rank, "scale": m.scale, "eps": cfg.norm_eps, "position": position, "sink": True,
        "names": {"q": "mix.q", "dkv": "mix.dkv", "dkv_norm": "mix.dkv.norm", "uk": "mix.uk", "uv": "mix.uv", "sink": "mix.sink", "o": "mix.o"}})


def _ffn(cfg: GevipelConfig, layer: GevipelLayer) -> PartSpec:
    mlp = layer.mlp
    return PartSpec("routed_experts", {
        "hidden_size": cfg.width, "n_experts": mlp.experts, "top": mlp.top, "expert_size": mlp.ff, "activation": "relu2",
        "score": "softmax", "correction": True, "normalize": False,
        "names": {"router": "mlp.router", "correction": "mlp.correction", "expert": "mlp.e{}", "up": "up", "down": "down"}})


def describe(cfg: GevipelConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        parts = dict(norm1=_norm(cfg, "norm1"), mixer=_mixer(cfg, layer), norm1b=_norm(cfg, "norm1b"))
        if layer.mlp is not None:
            parts.update(norm2=_norm(cfg, "norm2"), ffn=_ffn(cfg, layer), norm2b=_norm(cfg, "norm2b"))
        layers.append(LayerSpec(prefix=f"l{i}.", arrangement="sandwich_norm", parts=parts, params={"residual_scale": cfg.residual_mult}))
    schedule, entry = [], 0
    if any(again for _, again in cfg.runs()):
        layers.append(LayerSpec(prefix="loop.", arrangement="stream_add", parts={}))
    for i, again in cfg.runs():
        if again:
            schedule.append(ScheduleEntry(layer=len(cfg.layers), cache=entry))       # it keeps nothing: the entry stays empty
            entry += 1
        schedule.append(ScheduleEntry(layer=i, cache=entry))                          # every run of a layer has its own entry
        entry += 1
    return ModelSpec(
        name="Gevipel", hidden_size=cfg.width, vocab_size=cfg.vocab,
        embedding=PartSpec("token_embedding", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "embed",
                                               "scale": cfg.embedding_scale}),
        layers=tuple(layers), schedule=tuple(schedule), final_norm=_norm(cfg, "final.norm"),
        head=PartSpec("linear_head", {"vocab_size": cfg.vocab, "hidden_size": cfg.width, "name": "head"}),
        max_positions=cfg.max_positions)


register_architecture("Gevipel", GevipelConfig.from_dict, describe)
