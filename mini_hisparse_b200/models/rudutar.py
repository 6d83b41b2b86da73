"""Rudutar as data: the ModelSpec of a RudutarConfig and its registry entry.

The embedding's rows are normalised as they enter the stream; every layer is a pre-norm block.  The mixer is
sliding-window attention over convolved q, k and v with a bias by distance, a query temperature, a constant sink and an
output gate ("attention"), or sliding-window attention whose values are the keys as projected, with partial rotation and a
gate per head ("attention_2").  An attention layer with ``kv_from`` has no keys of its own: its run entry reads the cache of
the layer it names, which then keeps as many positions as the widest window among its readers.  The feed-forward is dense
with the exact gelu, or routed (sigmoid scores, groups by their two best, weights that are not renormalised, relu-squared
experts and a shared one), or missing.  Tensor names: embed, embed.norm, l<i>.{norm1, norm2, mix.*, mlp.*}, final.norm, head.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.rudutar import DenseFF, RudutarConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def rudutar_spec(cfg: RudutarConfig) -> ModelSpec:
    W = cfg.width
    norm = PartSpec.make("rmsnorm", width=W, eps=cfg.eps, weight_name="")
    keep = {}            # how many positions a cache keeps: the widest window among its owner and its readers
    for i, layer in enumerate(cfg.layers):
        owner = getattr(layer.mixer, "kv_from", None)
        owner = i if owner is None else owner
        keep[owner] = max(keep.get(owner, 0), layer.mixer.window)
    layers, order, entry_of = [], [], {}
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        entry = RunEntry(i)
        common = dict(hidden_size=W, q_heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale,
                      window=m.window, eps=cfg.eps)
        if layer.type == "attention":
            owner = i if m.kv_from is None else m.kv_from
            if m.kv_from is not None:
                entry = RunEntry(i, cache_of=entry_of[m.kv_from])
            mixer = PartSpec.make("sloped_attention", conv=m.conv, q_temp=m.q_temp, sink=0.0, keep=keep[owner],
                                  own_kv=m.kv_from is None, position=PartSpec.make("none"), **common)
        else:
            position = (PartSpec.make("rotary", head_dim=m.dim, theta=m.rot_base, rotary_dim=m.rot_dims, float64_table=True)
                        if m.rot_dims else PartSpec.make("none"))
            mixer = PartSpec.make("key_value_attention", position=position, **common)
        entry_of[i] = len(order)
        order.append(entry)
        parts = {"mixer_norm": norm, "mixer": mixer}
        if layer.mlp is not None:
            if isinstance(layer.mlp, DenseFF):
                ff = PartSpec.make("mlp_act", hidden_size=W, intermediate_size=layer.mlp.ff, activation="gelu")
            else:
                r = layer.mlp
                ff = PartSpec.make("routed_experts", hidden_size=W, experts=r.experts, top=r.top, expert_ff=r.expert_ff,
                                   shared_ff=r.shared_ff, group_count=r.group_count, group_keep=r.group_keep,
                                   score="sigmoid", group_score="two", normalise=False, factor=r.scale, form="relu2",
                                   shared_gate=False)
            parts.update({"ff_norm": norm, "feed_forward": ff})
        layers.append(LayerSpec.make(f"l{i}", "pre_norm", parts, {"mixer_norm": "norm1", "mixer": "mix", "ff_norm": "norm2",
                                                                  "feed_forward": "mlp"}))
    return ModelSpec(
        architecture="Rudutar", vocab_size=cfg.vocab, hidden_size=W,
        embedding=PartSpec.make("token_embedding", vocab_size=cfg.vocab, hidden_size=W, weight_name="",
                                norm=("norm", cfg.eps)),
        embedding_name="embed", layers=tuple(layers), order=tuple(order), final_norm=norm, final_norm_name="final.norm",
        head=PartSpec.make("lm_head", vocab_size=cfg.vocab, hidden_size=W, tied=False, weight_name=""), head_name="head",
    )


register_architecture("Rudutar", RudutarConfig, rudutar_spec, replace=True)
