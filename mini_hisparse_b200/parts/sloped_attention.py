"""Two kinds of sliding-window attention: over convolved q, k and v with a bias per head that grows with the distance
("sloped_attention"), and over keys that are the values too before they are normalised and rotated
("key_value_attention")."""
from __future__ import annotations

import torch

from ..kernels import api as K
from .base import CacheView, Product, StepContext
from .multimap_attention import _pad_rows
from .registry import register_mixer
from .sink_attention import SinkAttention
from .spec import ParamSpec, PartSpec, StateNeed


@register_mixer("sloped_attention")
class SlopedAttention(SinkAttention):
    """q = W_q h [q_heads x dim], k = W_k h [kv_heads x dim], v = W_v h [kv_heads x vdim], no biases.

    * q, k and v each pass a short causal convolution over time, one filter of ``conv`` taps per channel (the last tap is
      the current token's, zeros before the start of the sequence, no bias, no activation).
    * Every head's q and k is then RMS-normalised, with one weight [dim] each that the heads share.
    * ``q_temp`` = (coef, every): q at position p is multiplied by 1 + coef ln(floor((p + 1) / every) + 1) (None: not).
    * score_h(i, j) = (q_i . k_j) * scale - slope_h (i - j) over the last ``window`` positions (None: all), with
      slope_h = 2^(-slope_exponent (h + 1) / q_heads); nothing is rotated.
    * ``sink`` (a number, or None): the softmax's denominator has one more term exp(sink), the same for every head; it
      stands for no position.  Sink 0 adds one.
    * The heads' outputs are multiplied by sigmoid(W_g h), element by element, and projected by W_o.
    * ``own_kv`` False: no tensors for k and v; the layer reads the cache of another run entry (keys as cached: convolved
      and normalised; values as cached: convolved) with its own queries, window, slopes and gate.

    Convolutions, norms, temperature, scores, softmax and gate are float32; q and the cached keys and values have the
    compute dtype.  Beside the pages a request keeps the last conv - 1 projected rows in float32 (side memory "conv").
    Parameters: hidden_size, q_heads, kv_heads, dim, vdim, conv, scale, window, keep, eps, own_kv, position (a PartSpec that
    does not rotate), and optionally q_temp, sink, slope_exponent (default 8).  Tensors: q, k, v, q.conv, k.conv, v.conv,
    q.norm, k.norm, g, o.  The kernels and their choice by width are SinkAttention's.
    """

    MAX_TAPS = 16

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        if int(getattr(self.position, "rotary_dim", 0) or 0):
            raise ValueError("sloped_attention does not rotate: positions enter as distances")
        self.taps = int(spec["conv"])
        if not 1 <= self.taps <= self.MAX_TAPS:
            raise ValueError(f"the short convolution has 1 to {self.MAX_TAPS} taps")
        temp = spec.get("q_temp")
        self.q_temp = (float(temp[0]), float(temp[1])) if temp is not None else None
        if self.q_temp is not None and not self.q_temp[1] > 0:
            raise ValueError("the step of the query temperature must be positive")
        self.sink_value = spec.get("sink")
        self.slope_exponent = float(spec.get("slope_exponent", 8.0))
        self.channels = self.qw + (self.kw + self.vw if self.own_kv else 0)
        self.filters = self.slopes = None

    def kernel_modules(self):
        return super().kernel_modules() + ("headconv",)

    def side_needs(self):
        return {"conv": StateNeed(shape=(self.taps - 1, self.channels), dtype="float32")} if self.taps > 1 else {}

    def _names(self):
        return ("q", "k", "v") if self.own_kv else ("q",)

    def parameters(self):
        rows = {"q": self.qw, "k": self.kw, "v": self.vw}
        p = {"g": ParamSpec((self.ow, self.hidden)), "o": ParamSpec((self.hidden, self.ow))}
        for n in self._names():
            p[n] = ParamSpec((rows[n], self.hidden))
            p[n + ".conv"] = ParamSpec((rows[n], self.taps), role="vector", init=("normal", 0.0, 0.5))
            if n != "v":
                p[n + ".norm"] = ParamSpec((self.dk,), role="vector", init=("normal", 1.0, 0.1))
        return p

    def load(self, tensors):
        names = self._names()
        self.weight = _pad_rows(torch.cat([tensors[n] for n in names + ("g",)], 0))      # one product: [q | k | v | g]
        self.filters = torch.cat([tensors[n + ".conv"].float() for n in names], 0).t().contiguous()       # [taps, channels]
        self.o_weight = tensors["o"].contiguous()
        self.q_norm = tensors["q.norm"].float().contiguous()
        self.k_norm = tensors["k.norm"].float().contiguous() if self.own_kv else None
        h = torch.arange(1, self.nq + 1, dtype=torch.float64)
        dev = self.o_weight.device
        self.slopes = (2.0 ** (-self.slope_exponent * h / self.nq)).float().to(dev)
        self.sink = None if self.sink_value is None else torch.full((self.nq,), float(self.sink_value), device=dev)

    def forward(self, h, ctx: StepContext, cache: CacheView) -> Product:
        rt, ws, T = ctx.rt, ctx.ws, h.shape[0]
        if cache.writable != self.own_kv:
            raise ValueError("a sloped_attention layer with tensors for k and v owns its cache, one without reads another's")
        proj = rt.linear(h, self.weight, ws, "sl_proj", out_dtype=torch.float32)
        q = ws.get("sl_q", (T, self.qw), rt.dtype)
        kept = cache.sides["conv"].storage if self.taps > 1 else None
        K.head_conv_append(proj, self.filters, self.q_norm, self.k_norm, self.eps, kept, ctx, cache.meta["block_table"], q,
                           cache.storage, nq=self.nq, nkv=self.nkv, dk=self.dk, dv=self.dv, page_size=cache.page_size,
                           has_kv=self.own_kv, q_temp=self.q_temp)
        p = proj.tensor
        g0 = self.channels
        gate = dict(gate=(p[0] if proj.nsplit > 1 else p)[:, g0:g0 + self.ow], gate_nsplit=proj.nsplit,
                    gate_split_stride=proj.split_stride)
        attn = self._attend(q, gate, ctx, cache, sink=self.sink, slopes=self.slopes)
        return rt.linear(attn, self.o_weight, ws, "mix_out", out_dtype=torch.float32)


@register_mixer("key_value_attention")
class KeyValueAttention(SinkAttention):
    """q = W_q h + b_q [q_heads x dim], k = W_k h + b_k [kv_heads x dim]; the values are the keys as projected (with the
    bias, before norm and rotation), and there is no W_v.

    * q and k are each RMS-normalised as ONE vector spanning every head, and only then cut into heads and rotated by the
      position part.
    * score = (q . k) * scale over the last ``window`` positions (None: all); an ordinary softmax.
    * Head h's output is multiplied by sigmoid(W_g h)_h, one number per head, and the heads are projected by W_o.

    Biases, norms, angles, scores, softmax and gate are float32; q and the cached keys and values (both forms of the key)
    have the compute dtype.  Parameters: hidden_size, q_heads, kv_heads, dim, scale, window, eps, position (a PartSpec).
    Tensors: q, q.b, k, k.b, q.norm, k.norm, g, o.  The kernels and their choice by width are SinkAttention's.
    """

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        if not self.own_kv:
            raise ValueError("a key_value_attention layer owns its cache")
        if self.dv != self.dk:
            raise ValueError(f"values that are the keys are as wide as these: {self.dv} is not {self.dk}")
        self.bias = None

    def parameters(self):
        vec = dict(role="vector")
        return {"q": ParamSpec((self.qw, self.hidden)), "k": ParamSpec((self.kw, self.hidden)),
                "q.b": ParamSpec((self.qw,), init=("normal", 0.0, 0.1), **vec),
                "k.b": ParamSpec((self.kw,), init=("normal", 0.0, 0.1), **vec),
                "q.norm": ParamSpec((self.qw,), init=("normal", 1.0, 0.1), **vec),
                "k.norm": ParamSpec((self.kw,), init=("normal", 1.0, 0.1), **vec),
                "g": ParamSpec((self.nq, self.hidden)), "o": ParamSpec((self.hidden, self.ow))}

    def load(self, tensors):
        self.weight = _pad_rows(torch.cat([tensors[n] for n in ("q", "k", "g")], 0))     # one product: [q | k | g]
        self.bias = torch.cat((tensors["q.b"].float(), tensors["k.b"].float())).contiguous()
        self.o_weight = tensors["o"].contiguous()
        self.q_norm, self.k_norm = tensors["q.norm"].float().contiguous(), tensors["k.norm"].float().contiguous()

    def forward(self, h, ctx: StepContext, cache: CacheView) -> Product:
        rt, ws, T = ctx.rt, ctx.ws, h.shape[0]
        if not cache.writable:
            raise ValueError("a key_value_attention layer owns its cache")
        proj = rt.linear(h, self.weight, ws, "kv_proj", out_dtype=torch.float32)
        p = proj.tensor
        q = ws.get("kv_q", (T, self.qw), rt.dtype)
        rdim = int(getattr(self.position, "rotary_dim", 0) or 0)
        K.qknorm_rope_append(p, self.q_norm, self.k_norm, self.eps, ctx.positions, ctx.tok_seg, cache.meta["block_table"],
                             self.position.inv_freq, rdim, q, cache.storage, nq=self.nq, nkv=self.nkv, dk=self.dk,
                             dv=self.dv, page_size=cache.page_size, nsplit=proj.nsplit, split_stride=proj.split_stride,
                             status=ctx.status, bias=self.bias, v_from_k=True)
        g0 = self.qw + self.kw
        gate = dict(gate=(p[0] if proj.nsplit > 1 else p)[:, g0:g0 + self.nq], gate_nsplit=proj.nsplit,
                    gate_split_stride=proj.split_stride, gate_per_head=True)
        attn = self._attend(q, gate, ctx, cache)
        return rt.linear(attn, self.o_weight, ws, "mix_out", out_dtype=torch.float32)
