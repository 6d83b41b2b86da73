"""The selective scan (Mamba): a diagonal linear recurrence over a float32 state whose step size, input vector and output
vector are made from the input row."""
from __future__ import annotations

import math

import torch

from ..kernels import api as K
from .base import CacheView, Mixer, Product, StepContext
from .multimap_attention import _pad_rows
from .registry import register_mixer
from .spec import ParamSpec, PartSpec, StateNeed


@register_mixer("selective_scan")
class SelectiveScan(Mixer):
    """[x | z] = W_in h, both ``inner`` wide.

    * x passes a causal convolution over time, one filter of ``conv`` taps and a bias per channel (the last tap is the
      current token's, zeros before the start of the sequence), and silu.
    * [dt | B | C] = W_x x with dt_rank, ``state`` and ``state`` numbers; dt <- softplus(W_dt dt + b), one per channel.
    * Per channel c and state n, with A = -exp(A_log):  S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;
      y_c = sum_n S[c, n] C_n + D_c x_c  (y sees the token's own write).
    * The output is W_o (y * silu(z)), times ``out_scale``.

    Per request: the state [inner x state] and the convolution's last conv - 1 inputs, both float32, in one slot.  The
    convolution, dt, the decays, the recurrence and the gate are float32; the matrix products' operands have the compute
    dtype.  Parameters: hidden_size, inner, state, dt_rank, conv, and optionally out_scale.
    Tensors: in, conv, conv.b, x, dt, dt.b, A_log, D, o.
    """

    #: up to this many tokens in a step, each segment at most FUSE_SEGMENT long, dt's product is taken inside the scan
    FUSE_TOKENS, FUSE_SEGMENT = 64, 16

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.hidden, self.inner = int(spec["hidden_size"]), int(spec["inner"])
        self.states, self.rank = int(spec["state"]), int(spec["dt_rank"])
        self.taps = int(spec["conv"])
        self.out_scale = float(spec.get("out_scale", 1.0))
        if min(self.inner, self.states, self.rank) < 1:
            raise ValueError("a selective scan has at least one channel, one state and a step of rank one")
        if self.states > K.SELECTIVE_STATES:
            raise ValueError(f"the selective scan takes up to {K.SELECTIVE_STATES} states per channel")
        if not 1 <= self.taps <= 16:
            raise ValueError("the short convolution has 1 to 16 taps")
        self.weight = self.x_weight = self.dt_weight = self.o_weight = None
        self.filters = self.conv_bias = self.dt_bias = self.A2 = self.D = None

    def kernel_modules(self):
        return ("timeconv", "selscan")

    def cache_need(self):
        return StateNeed(shape=(self.inner * (self.states + self.taps - 1),), dtype="float32")

    def parameters(self):
        vec = dict(role="vector")
        return {"in": ParamSpec((2 * self.inner, self.hidden)),
                "conv": ParamSpec((self.inner, self.taps), init=("normal", 0.0, 0.5), **vec),
                "conv.b": ParamSpec((self.inner,), init=("normal", 0.0, 0.1), **vec),
                "x": ParamSpec((self.rank + 2 * self.states, self.inner)),
                "dt": ParamSpec((self.inner, self.rank)),
                "dt.b": ParamSpec((self.inner,), init=("normal", -2.0, 1.0), **vec),
                "A_log": ParamSpec((self.inner, self.states), init=("normal", 0.0, 1.0), **vec),
                "D": ParamSpec((self.inner,), init=("normal", 1.0, 0.1), **vec),
                "o": ParamSpec((self.hidden, self.inner))}

    def load(self, tensors):
        self.weight = _pad_rows(tensors["in"])                                           # [x | z]
        self.x_weight = _pad_rows(tensors["x"])                                          # [dt | B | C]
        # dt's matrix with zero columns up to a multiple of 8, as its product's other operand is padded
        self.rank_pad = -(-self.rank // 8) * 8
        dt = tensors["dt"]
        self.dt_weight = torch.cat((dt, dt.new_zeros(self.inner, self.rank_pad - self.rank)), 1).contiguous()
        self.o_weight = tensors["o"].contiguous()
        self.filters = tensors["conv"].float().t().contiguous()                          # [taps, inner]
        self.conv_bias, self.dt_bias = tensors["conv.b"].float().contiguous(), tensors["dt.b"].float().contiguous()
        self.A2 = (-torch.exp(tensors["A_log"].float()) * math.log2(math.e)).contiguous()
        self.D = tensors["D"].float().contiguous()

    def take_input(self) -> torch.Tensor:
        """Give up the input projection (a mixer that stacks several of them runs the product itself)."""
        w, self.weight = self.weight, None
        return w

    def forward(self, h, ctx: StepContext, cache: CacheView) -> Product:
        proj = ctx.rt.linear(h, self.weight, ctx.ws, "ss_proj", out_dtype=torch.float32)
        return self.forward_projected(proj, 0, ctx, cache, "mix_out")

    def forward_projected(self, proj: Product, col0: int, ctx: StepContext, cache: CacheView, name: str) -> Product:
        """From the input projection's columns col0 ...: convolution, recurrence, W_o."""
        rt, ws, T = ctx.rt, ctx.ws, proj.tensor.shape[-2]
        C, N = self.inner, self.states
        slots = cache.storage                                            # [slots, state | kept inputs]
        x32 = ws.get("ss_x32", (T, C), torch.float32)
        x = x32 if rt.dtype == torch.float32 else ws.get("ss_x", (T, C), rt.dtype)
        K.product_conv(proj, col0, self.filters, self.conv_bias, slots[:, C * N:] if self.taps > 1 else None, ctx, x,
                       out32=None if x is x32 else x32, writable=cache.writable)
        low = rt.linear(x, self.x_weight, ws, "ss_low", out_dtype=torch.float32)
        y = ws.get("ss_y", (T, C), rt.dtype)
        common = dict(scale=self.out_scale, writable=cache.writable)
        if T <= self.FUSE_TOKENS and ctx.longest <= self.FUSE_SEGMENT:
            K.selective_scan(proj, col0 + C, low, low, self.rank, x32, self.dt_bias, self.A2, self.D, slots, ctx, y,
                             dt_weight=self.dt_weight, rank=self.rank, **common)
        else:
            dt_in = ws.get("ss_dt_in", (T, self.rank_pad), rt.dtype)
            bc = ws.get("ss_bc", (T, 2 * N), torch.float32)
            K.selective_split(low, self.rank, N, dt_in, bc)
            dt = rt.linear(dt_in, self.dt_weight, ws, "ss_dt", out_dtype=torch.float32)
            K.selective_scan(proj, col0 + C, dt, Product(bc), 0, x32, self.dt_bias, self.A2, self.D, slots, ctx, y, **common)
        return rt.linear(y, self.o_weight, ws, name, out_dtype=torch.float32)
