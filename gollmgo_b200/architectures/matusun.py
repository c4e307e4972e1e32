"""Matusun as a ModelSpec: several residual streams that every sublayer reads through a learned contraction and
writes through a learned mixing (hyper-connections, RMS norms before the sublayers), two kinds of mixer listed
layer by layer (grouped-query attention with one norm over each whole projection of q and k, rotary positions and
a sliding window; a selective scan of the Mamba-1 kind), a mixture of squared-ReLU experts (softmax scores, a
correction of the choice, identity experts) beside a shared expert, a run of layers that is repeated with the same
weights and caches of its own per pass, an RMS norm and the embedding table as the head.
Tensor names: layer i's start with "l<i>.", the mixer's with "l<i>.mix.", the feed-forward's with "l<i>.mlp.", the
streams' with "l<i>.hc1." and "l<i>.hc2."; the norms are "l<i>.norm1" and "l<i>.norm2".
"""
from __future__ import annotations

from ..config import register_architecture
from ..config.matusun_config import MatusunConfig, RowNormedAttentionConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, looped_run_order


def _mixer(cfg: MatusunConfig, m) -> PartSpec:
    if isinstance(m, RowNormedAttentionConfig):
        position = PartSpec("none")
        if m.rot is not None:
            position = PartSpec("rope", {"head_dim": m.dim, "rotary_dim": m.rot[1], "theta": m.rot[0]})
        return PartSpec("attention", {"hidden_size": cfg.width, "num_heads": m.heads, "num_kv_heads": m.kv_heads,
                                      "head_dim": m.dim, "v_head_dim": m.vdim, "window": m.window, "scale": m.scale,
                                      "position": position, "row_norm": cfg.eps, "names": ("q", "k", "v", "o")})
    return PartSpec("mamba1", {"hidden_size": cfg.width, "inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "conv": m.conv})


def _feed_forward(cfg: MatusunConfig, f):
    if f is None:
        return None
    shared = None
    if f.shared_ff is not None:
        shared = PartSpec("mlp", {"hidden_size": cfg.width, "intermediate_size": f.shared_ff, "activation": "relu2",
                                  "names": ("up", "down")})
    return PartSpec("moe", {"hidden_size": cfg.width, "intermediate_size": f.ff, "experts": f.experts, "top": f.top,
                            "gated": False, "activation": "relu2", "router_bias": False, "router_weigh": "softmax_all",
                            "router_scale": f.scale, "correction": True, "identity": f.identity, "shared": shared})


def matusun_spec(cfg: MatusunConfig) -> ModelSpec:
    norm = PartSpec("rmsnorm", {"size": cfg.width, "eps": cfg.eps})
    block = PartSpec("streams", {"streams": cfg.streams, "names": ("hc1", "hc2")})
    layers, ignorable = [], []
    for i, lc in enumerate(cfg.layers):
        p = f"l{i}."
        ff = _feed_forward(cfg, lc.mlp)
        if ff is None:
            ignorable += [p + "norm2", p + "hc2.*"]
        layers.append(LayerSpec(block, _mixer(cfg, lc.mixer), ff, norm, norm if ff is not None else None,
                                mixer_prefix=p + "mix.", ffn_prefix=p + "mlp.", mixer_norm_name=p + "norm1",
                                ffn_norm_name=p + "norm2", block_prefix=p))
    lp = cfg.loop
    order = looped_run_order(len(layers), lp.start, lp.stop, lp.times) if lp is not None else looped_run_order(len(layers))
    return ModelSpec(architecture="Matusun", vocab_size=cfg.vocab, hidden_size=cfg.width, layers=tuple(layers),
                     run_order=order, final_norm=norm, tie_embeddings=True, embed_name="embed",
                     final_norm_name="final.norm", head_name="head", max_positions=cfg.max_position_embeddings,
                     eos_token_ids=cfg.eos_token_ids, bos_token_id=cfg.bos_token_id, ignorable_tensors=tuple(ignorable))


register_architecture("Matusun", MatusunConfig.from_dict, matusun_spec)
