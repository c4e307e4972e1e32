"""Rimidra as a ModelSpec: parallel blocks (one RMS norm whose weight is stored around zero; mixer and
feed-forward read its output and are both added to the stream), two kinds of mixer listed layer by layer
(grouped-query attention without rotation, with a bias by distance, a sliding window, a sink in the softmax
and a query temperature; retention with fixed decays and rotary positions), a GELU-gated feed-forward or a
mixture of SiLU-gated experts (sigmoid scores that multiply the experts' input, a gated shared expert), an
RMS norm and an untied head.  A layer may use another layer's tensors with a cache of its own: such a layer
is one more entry of the run order, not a layer of the spec.
Tensor names: layer i's start with "l<i>.", the mixer's with "l<i>.mix.", the feed-forward's with
"l<i>.mlp."; the norm is "l<i>.norm1".
"""
from __future__ import annotations

from ..config import register_architecture
from ..config.rimidra_config import RimidraConfig, SlopedAttentionConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry

_GATED = ("gate", "up", "down")


def _mixer(cfg: RimidraConfig, m) -> PartSpec:
    if isinstance(m, SlopedAttentionConfig):
        return PartSpec("attention", {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads,
                                      "head_dim": m.dim, "v_head_dim": m.vdim, "window": m.window, "scale": m.scale,
                                      "position": PartSpec("none"), "distance_bias": True, "sink": True,
                                      "temperature": m.q_temp, "names": ("q", "k", "v", "o")})
    position = PartSpec("none")
    if m.rot is not None:
        position = PartSpec("rope", {"head_dim": m.dim, "rotary_dim": m.rot[1], "theta": m.rot[0]})
    return PartSpec("retention", {"hidden_size": cfg.width, "num_heads": m.heads, "head_dim": m.dim, "v_head_dim": m.vdim,
                                  "decay": m.decay, "position": position, "eps": cfg.eps})


def _feed_forward(cfg: RimidraConfig, f):
    if f is None:
        return None
    if f.kind == "dense":
        return PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": f.ff, "activation": "gelu_tanh",
                                      "names": _GATED})
    shared = None
    if f.shared_ff is not None:
        shared = PartSpec("gated_mlp", {"hidden_size": cfg.width, "intermediate_size": f.shared_ff, "activation": "silu",
                                        "names": _GATED})
    return PartSpec("moe", {"hidden_size": cfg.width, "intermediate_size": f.ff, "experts": f.experts, "top": f.top,
                            "router_bias": False, "router_weigh": "sigmoid", "weigh_input": True, "shared": shared,
                            "shared_gate": shared is not None})


def rimidra_spec(cfg: RimidraConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.eps, "offset": True})
    layers, place = [], {}
    for i, lc in enumerate(cfg.layers):
        if lc.weights_of is not None:
            continue
        p = f"l{i}."
        place[i] = len(layers)
        layers.append(LayerSpec(PartSpec("parallel", {}), _mixer(cfg, lc.mixer), _feed_forward(cfg, lc.mlp), norm, None,
                                mixer_prefix=p + "mix.", ffn_prefix=p + "mlp.", mixer_norm_name=p + "norm1", block_prefix=p))
    order = tuple(RunEntry(place[i if lc.weights_of is None else lc.weights_of], i) for i, lc in enumerate(cfg.layers))
    return ModelSpec(architecture="Rimidra", vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers),
                     run_order=order, final_norm=norm, tie_embeddings=False, embed_name="embed",
                     final_norm_name="final.norm", head_name="head", max_positions=cfg.max_position_embeddings,
                     eos_token_ids=cfg.eos_token_ids, bos_token_id=cfg.bos_token_id)


register_architecture("Rimidra", RimidraConfig.from_dict, rimidra_spec)
