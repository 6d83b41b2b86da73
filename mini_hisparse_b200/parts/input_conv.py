"""A short causal convolution in front of a sublayer: h <- h + conv(h)."""
from __future__ import annotations

from ..kernels import api as K
from .base import Part, StepContext
from .registry import register_input_conv
from .spec import ParamSpec, PartSpec


@register_input_conv("causal_conv")
class CausalConv(Part):
    """h <- h + conv(h), conv(h)_t = sum_j w[:, j] h_(t - taps + 1 + j) per channel, zeros before the start of the
    sequence, no bias.  Per request the last taps - 1 inputs are kept in float32; whoever holds the part hands them to
    forward() ([slots, taps - 1, width]).  Parameters: width, taps, weight_name.  Tensor [width, taps].

    Behind a norm that works element by element (a norm with ``forward_conv``) the convolution rides in the norm's kernel;
    behind any other it is a kernel of its own on the normalised rows.
    """

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.width, self.taps = int(spec["width"]), int(spec["taps"])
        self.weight_name = spec.get("weight_name", "weight")
        if not 1 <= self.taps <= 16:
            raise ValueError("an input convolution has 1 to 16 taps")
        self.filters = None

    def kernel_modules(self):
        return ("timeconv",)

    @property
    def kept_shape(self) -> tuple[int, int]:
        return (self.taps - 1, self.width)

    def parameters(self):
        return {self.weight_name: ParamSpec((self.width, self.taps), role="vector", init=("normal", 0.0, 0.3))}

    def load(self, tensors):
        self.filters = tensors[self.weight_name].float().t().contiguous()               # [taps, width]

    def forward(self, h, ctx: StepContext, kept, name="h_conv", writable=True):
        out = ctx.ws.get(name, tuple(h.shape), h.dtype)
        K.rows_conv(h, self.filters, kept, ctx, out, writable=writable)
        return out
