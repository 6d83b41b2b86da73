"""minGRU: one number per channel and request, blended with a candidate; gate and candidate are functions of the input row."""
from __future__ import annotations

import torch

from ..kernels import api as K
from .base import CacheView, Mixer, Product, StepContext
from .multimap_attention import _pad_rows
from .registry import register_mixer
from .spec import ParamSpec, PartSpec, StateNeed


@register_mixer("mingru")
class MinGRU(Mixer):
    """z = sigmoid(W_z h + b_z), u = W_x h + b_x, candidate c = u + 1/2 where u >= 0 and sigmoid(u) where u < 0, all
    ``width`` wide;  S <- (1 - z) S + z c  over a float32 state that starts at zero;  W_o (S * silu(W_g h)).

    Everything between the two projections is float32.  Parameters: hidden_size, width.
    Tensors: z, z.b, x, x.b, g, o.
    """

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.hidden, self.width = int(spec["hidden_size"]), int(spec["width"])
        if self.width < 1:
            raise ValueError("a minGRU layer has at least one channel")
        self.weight = self.o_weight = self.z_bias = self.x_bias = None

    def kernel_modules(self):
        return ("selscan",)

    def cache_need(self):
        return StateNeed(shape=(self.width,), dtype="float32")

    def parameters(self):
        W, H = self.width, self.hidden
        bias = dict(role="vector", init=("normal", 0.0, 0.5))
        return {"z": ParamSpec((W, H)), "z.b": ParamSpec((W,), **bias), "x": ParamSpec((W, H)), "x.b": ParamSpec((W,), **bias),
                "g": ParamSpec((W, H)), "o": ParamSpec((H, W))}

    def load(self, tensors):
        self.weight = _pad_rows(torch.cat([tensors[n] for n in ("z", "x", "g")], 0))           # [z | x | g]
        self.z_bias, self.x_bias = tensors["z.b"].float().contiguous(), tensors["x.b"].float().contiguous()
        self.o_weight = tensors["o"].contiguous()

    def forward(self, h, ctx: StepContext, cache: CacheView) -> Product:
        rt, ws, T, W = ctx.rt, ctx.ws, h.shape[0], self.width
        proj = rt.linear(h, self.weight, ws, "gru_proj", out_dtype=torch.float32)
        y = ws.get("gru_y", (T, W), rt.dtype)
        K.mingru_scan(proj, 0, W, 2 * W, self.z_bias, self.x_bias, cache.storage, ctx, y, writable=cache.writable)
        return rt.linear(y, self.o_weight, ws, "mix_out", out_dtype=torch.float32)
