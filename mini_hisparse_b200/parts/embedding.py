"""Token embedding and output head."""
from __future__ import annotations

import torch

from ..kernels import api as K
from .base import Part, Product, StepContext
from .registry import EMBEDDINGS, HEADS
from .spec import ParamSpec, PartSpec


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Part):
    """x = table[tokens] (mini_hisparse/model.py:86,166), times ``scale`` if the spec gives one (the
    reference has none); output is the float32 residual.  ``weight_name``: the tensor's local name
    ("" if the prefix alone names it).  With ``copy`` the rows are also left in the compute dtype as
    ctx.extras["x_copy"], for a first block that reads the stream without normalising it.  With
    ``keep`` = (name, row width, first column) the rows are also left, in the compute dtype, in those
    columns of a matrix ctx.extras[name] [T, row width], for a later part that reads the embedding
    output again (the input of a pass over repeated layers).  With ``norm`` = (tensor's local name, eps) the row
    enters the stream as rms(row) * weight, in the gather's kernel (then without a scale and a copy)."""

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.norm = spec.get("norm")
        self.norm_weight = None
        self.vocab = int(spec["vocab_size"])
        self.width = int(spec["hidden_size"])
        self.scale = float(spec.get("scale", 1.0))
        self.copy = bool(spec.get("copy", False))
        self.keep = spec.get("keep")
        self.weight_name = spec.get("weight_name", "weight")
        if self.norm and (self.scale != 1.0 or self.copy):
            raise ValueError("an embedding that normalises its rows takes no scale and keeps no copy")
        self.weight = None

    def kernel_modules(self):
        return ("mixparts",) if self.keep else ()

    def parameters(self):
        p = {self.weight_name: ParamSpec((self.vocab, self.width))}
        if self.norm:
            p[self.norm[0]] = ParamSpec((self.width,), role="vector", init=("normal", 1.0, 0.1))
        return p

    def load(self, tensors):
        self.weight = tensors[self.weight_name].contiguous()
        if self.norm:
            self.norm_weight = tensors[self.norm[0]].contiguous()

    def forward(self, ctx: StepContext) -> torch.Tensor:
        x = self._forward(ctx)
        if self.keep:
            name, ld, col0 = self.keep
            kept = ctx.ws.get(name, (ctx.T, int(ld)), ctx.rt.dtype)
            K.stream_pack(x, kept, int(col0))
            ctx.extras[name] = kept
        return x

    def _forward(self, ctx: StepContext) -> torch.Tensor:
        x = ctx.ws.get("residual", (ctx.T, self.width), torch.float32)
        copy = None
        if self.norm:
            K.embed_norm(self.weight, self.norm_weight, float(self.norm[1]), ctx.tokens, x, status=ctx.status)
            return x
        if self.copy and ctx.rt.dtype != torch.float32:
            copy = ctx.ws.get("x_copy", (ctx.T, self.width), ctx.rt.dtype)
        K.embed(self.weight, ctx.tokens, x, status=ctx.status, scale=self.scale, copy=copy)
        if self.copy:
            ctx.extras["x_copy"] = x if copy is None else copy
        return x


@EMBEDDINGS.register("stream_input")
class StreamInput(Part):
    """A part of the model as a whole that replaces the residual stream by a product of itself and the
    embedding output:  x <- W [x ; x0]  with W [width, 2 width] (x's columns first).  It runs where the
    run order says (RunEntry.before), e.g. at the start of every pass over repeated layers.

    The embedding leaves x0 in the right half of ctx.extras[``buffer``] [T, 2 width] (TokenEmbedding's
    ``keep``); this part writes the stream, with everything still pending added, into the left half,
    leaves the stream at ZERO and returns the product as pending, so that the next norm's pass over the
    stream adds it (0 + W [x ; x0]) like any other product, split-K parts included."""

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.width = int(spec["width"])
        self.buffer = spec.get("buffer", "stream_cat")
        self.weight_name = spec.get("weight_name", "in")
        self.weight = None

    def kernel_modules(self):
        return ("mixparts",)

    def parameters(self):
        return {self.weight_name: ParamSpec((self.width, 2 * self.width))}

    def load(self, tensors):
        self.weight = tensors[self.weight_name].contiguous()

    def forward_stream(self, x, pending: Product | None, ctx: StepContext, turn: int = 0):
        cat = ctx.extras.get(self.buffer)
        if cat is None:
            raise RuntimeError(f"the embedding did not keep its output in {self.buffer!r}")
        K.stream_pack(x, cat, 0, delta=pending, delta2=pending.also if pending is not None else None, zero=True)
        return x, ctx.rt.linear(cat, self.weight, ctx.ws, "stream_in", out_dtype=torch.float32)


@EMBEDDINGS.register("pass_input")
class PassInput(Part):
    """A part of the model as a whole that opens every pass over repeated layers:  x <- x + x0 (not before the
    first pass), then x <- x + step[turn], with x0 the embedding output (the table's row times the embedding's
    scale, gathered again rather than kept) and ``step`` [times, width] one stored vector per pass.  Everything
    pending is added in the same kernel, in float32.  Parameters: width, times, weight_name."""

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.width, self.times = int(spec["width"]), int(spec["times"])
        self.weight_name = spec.get("weight_name", "step")
        self.step = None
        self._embedding = None

    def kernel_modules(self):
        return ("timeconv",)

    def parameters(self):
        return {self.weight_name: ParamSpec((self.times, self.width), role="vector", init=("normal", 0.0, 0.1))}

    def load(self, tensors):
        self.step = tensors[self.weight_name].float().contiguous()

    def tie(self, embedding: TokenEmbedding):
        self._embedding = embedding

    def forward_stream(self, x, pending: Product | None, ctx: StepContext, turn: int = 0):
        if pending is not None:
            pending = pending.settle_also(x)
        e = self._embedding
        K.stream_shift(x, self.step[turn], delta=pending, table=e.weight if turn else None, tokens=ctx.tokens,
                       scale=e.scale)
        return x, None


@EMBEDDINGS.register("token_table")
class TokenTable(Part):
    """A table [vocab, width] that other parts index by token id (a model-level part: ModelSpec.shared)."""

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.vocab = int(spec["vocab_size"])
        self.width = int(spec["width"])
        self.weight_name = spec.get("weight_name", "weight")
        self.weight = None

    def parameters(self):
        return {self.weight_name: ParamSpec((self.vocab, self.width))}

    def load(self, tensors):
        self.weight = tensors[self.weight_name].contiguous()


@HEADS.register("lm_head")
class LMHead(Part):
    """logits = h W^T in float32, no bias (mini_hisparse/model.py:96,181).  With ``tied`` the
    embedding table is the weight and the checkpoint holds no lm_head tensor.  With ``softcap`` c the logits
    are capped smoothly: logits <- c tanh(logits / c), in float32."""

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.vocab = int(spec["vocab_size"])
        self.width = int(spec["hidden_size"])
        self.tied = bool(spec["tied"])
        self.softcap = float(spec.get("softcap") or 0.0)
        self.weight_name = spec.get("weight_name", "weight")
        self.weight = None

    def parameters(self):
        if self.tied:
            return {self.weight_name: ParamSpec((self.vocab, self.width), optional=True)}
        return {self.weight_name: ParamSpec((self.vocab, self.width))}

    def load(self, tensors):
        if not self.tied:
            self.weight = tensors[self.weight_name].contiguous()

    def tie(self, embedding: TokenEmbedding):
        self.weight = embedding.weight

    def kernel_modules(self):
        return ("gateparts",) if self.softcap else ()

    def forward(self, h: torch.Tensor, ctx: StepContext) -> torch.Tensor:
        logits = ctx.rt.linear(h, self.weight, ctx.ws, "logits", out_dtype=torch.float32, allow_split=False).matrix
        if self.softcap:
            K.softcap_rows(logits, self.softcap)
        return logits
