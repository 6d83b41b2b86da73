"""Zetenex as data: the ModelSpec of a ZetenexConfig and its registry entry.

Every layer is a pre-norm block whose norm is a dynamic tanh and whose sublayers each read h + conv(h), a short causal
convolution of the normalised stream.  The mixer is a minGRU ("mingru") or two mixers side by side ("parallel"):
attention over unit q and k with a position-dependent query temperature and a gate per head, and a selective scan, each
with a factor.  The feed-forward is down(gelu_tanh(up h)).  A run of layers may repeat: every pass has caches and states
of its own (a run entry each) and opens with x <- x + embedding output (not the first) and x <- x + step[pass].  The head
is the embedding table.  Tensor names: embed, loop.step, l<i>.{norm1, norm2, canon1, canon2, mix.*, mlp.{up,down}},
final.norm.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.zetenex import MinGRUMixer, ZetenexConfig
from ..parts.spec import LayerSpec, ModelSpec, PartSpec, RunEntry


def zetenex_spec(cfg: ZetenexConfig) -> ModelSpec:
    W = cfg.width
    norm = PartSpec.make("dyt", width=W, weight_name="")
    conv = PartSpec.make("causal_conv", width=W, taps=cfg.taps, weight_name="")
    layers = []
    for i, layer in enumerate(cfg.layers):
        m = layer.mixer
        if isinstance(m, MinGRUMixer):
            mixer = PartSpec.make("mingru", hidden_size=W, width=m.width)
        else:
            a, b = m.left, m.right
            mixer = PartSpec.make(
                "side_by_side",
                left=PartSpec.make("unit_attention", hidden_size=W, q_heads=a.heads, kv_heads=a.kv_heads, dim=a.dim,
                                   vdim=a.vdim, scale=a.scale, eps=cfg.eps, q_temp=a.q_temp, out_scale=m.left_scale,
                                   position=PartSpec.make("none")),
                right=PartSpec.make("selective_scan", hidden_size=W, inner=b.inner, state=b.state, dt_rank=b.dt_rank,
                                    conv=b.conv, out_scale=m.right_scale))
        parts = {"mixer_norm": norm, "mixer_conv": conv, "mixer": mixer}
        if layer.ff is not None:
            parts.update({"ff_norm": norm, "ff_conv": conv,
                          "feed_forward": PartSpec.make("mlp_act", hidden_size=W, intermediate_size=layer.ff,
                                                        activation="gelu_tanh")})
        layers.append(LayerSpec.make(f"l{i}", "pre_norm_conv", parts,
                                     {"mixer_norm": "norm1", "mixer_conv": "canon1", "mixer": "mix", "ff_norm": "norm2",
                                      "ff_conv": "canon2", "feed_forward": "mlp"}))
    n, loop = len(cfg.layers), cfg.loop
    shared = ()
    if loop is None:
        order = [RunEntry(i) for i in range(n)]
    else:
        order = [RunEntry(i) for i in range(loop.start)]
        for turn in range(loop.times):           # the same weights, caches and states of its own for every pass
            order += [RunEntry(i, before="loop" if i == loop.start else None, turn=turn)
                      for i in range(loop.start, loop.stop)]
        order += [RunEntry(i) for i in range(loop.stop, n)]
        shared = (("loop", PartSpec.make("pass_input", width=W, times=loop.times, weight_name="step"), "loop"),)
    return ModelSpec(
        architecture="Zetenex", vocab_size=cfg.vocab, hidden_size=W,
        embedding=PartSpec.make("token_embedding", vocab_size=cfg.vocab, hidden_size=W, weight_name="",
                                scale=cfg.embedding_scale),
        embedding_name="embed", layers=tuple(layers), order=tuple(order), final_norm=norm, final_norm_name="final.norm",
        head=PartSpec.make("lm_head", vocab_size=cfg.vocab, hidden_size=W, tied=True, weight_name="weight"),
        head_name="head", shared=shared,
    )


register_architecture("Zetenex", ZetenexConfig, zetenex_spec, replace=True)
