"""Grouped-query attention over unit q and k with a temperature that grows with the position and a gate per head."""
from __future__ import annotations

import torch

from ..kernels import api as K
from .base import CacheView, Product, StepContext
from .multimap_attention import _pad_rows
from .registry import register_mixer
from .sink_attention import SinkAttention
from .spec import ParamSpec, PartSpec


@register_mixer("unit_attention")
class UnitAttention(SinkAttention):
    """q = W_q h [q_heads x dim], k = W_k h [kv_heads x dim], v = W_v h [kv_heads x vdim], no biases.

    * Every head's q and k is divided by its root mean square over dim (no weight).
    * ``q_temp`` = (coef, every): q at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1)
      (None: not at all).  There is no other trace of the position in q and k, unless ``position`` rotates.
    * score = (q . k) * scale, a causal softmax over every earlier position (the last ``window``, if there is one).
    * Head h's output is multiplied by sigmoid(W_g h)_h, one number per head, and the heads are projected by W_o.
    * ``out_scale``: a factor on the whole result; it rides on the values as they are stored, in float32.

    Norms, the temperature, scores, softmax and the gate are float32; q and the cached keys and values have the compute
    dtype.  Parameters: hidden_size, q_heads, kv_heads, dim, vdim, scale, eps, position (a PartSpec), and optionally
    window, q_temp, out_scale.  Tensors: q, k, v, g, o.  The kernels and their choice by width are SinkAttention's.
    """

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        if not self.own_kv:
            raise ValueError("a unit_attention layer owns its cache")
        temp = spec.get("q_temp")
        self.q_temp = (float(temp[0]), float(temp[1])) if temp is not None else None
        if self.q_temp is not None and not self.q_temp[1] > 0:
            raise ValueError("the step of the query temperature must be positive")
        self.out_scale = float(spec.get("out_scale", 1.0))

    def plan_key(self):
        return ("unit_attention", self.nq, self.nkv, self.window)

    def parameters(self):
        return {"q": ParamSpec((self.qw, self.hidden)), "k": ParamSpec((self.kw, self.hidden)),
                "v": ParamSpec((self.vw, self.hidden)), "g": ParamSpec((self.nq, self.hidden)),
                "o": ParamSpec((self.hidden, self.ow))}

    def load(self, tensors):
        self.weight = _pad_rows(torch.cat([tensors[n] for n in ("q", "k", "v", "g")], 0))      # [q | k | v | g]
        self.o_weight = tensors["o"].contiguous()

    def take_input(self) -> torch.Tensor:
        """Give up the stacked input projection (a mixer that stacks several of them runs the product itself)."""
        w, self.weight = self.weight, None
        return w

    def forward(self, h, ctx: StepContext, cache: CacheView) -> Product:
        proj = ctx.rt.linear(h, self.weight, ctx.ws, "ua_proj", out_dtype=torch.float32)
        return self.forward_projected(proj, 0, ctx, cache, "mix_out")

    def forward_projected(self, proj: Product, col0: int, ctx: StepContext, cache: CacheView, name: str) -> Product:
        """From the input projection's columns col0 ...: q, k and v into place, attention, W_o."""
        rt, ws, T = ctx.rt, ctx.ws, proj.tensor.shape[-2]
        if not cache.writable:
            raise ValueError("a unit_attention layer owns its cache")
        p = proj.tensor[..., col0:]
        q = ws.get("ua_q", (T, self.qw), rt.dtype)
        rdim = int(getattr(self.position, "rotary_dim", 0) or 0)
        K.qknorm_rope_append(p, None, None, self.eps, ctx.positions, ctx.tok_seg, cache.meta["block_table"],
                             self.position.inv_freq, rdim, q, cache.storage, nq=self.nq, nkv=self.nkv, dk=self.dk,
                             dv=self.dv, page_size=cache.page_size, nsplit=proj.nsplit, split_stride=proj.split_stride,
                             status=ctx.status, per_head=True, q_temp=self.q_temp, v_scale=self.out_scale)
        g0 = self.qw + self.kw + self.vw
        gate = dict(gate=(p[0] if proj.nsplit > 1 else p)[:, g0:g0 + self.nq], gate_nsplit=proj.nsplit,
                    gate_split_stride=proj.split_stride, gate_per_head=True)
        attn = self._attend(q, gate, ctx, cache)
        return rt.linear(attn, self.o_weight, ws, name, out_dtype=torch.float32)
