"""Two mixers side by side: both read the same input, their results are added."""
from __future__ import annotations

import torch

from ..kernels import api as K
from .base import CacheView, Mixer, Product, StepContext
from .multimap_attention import _pad_rows
from .registry import MIXERS, register_mixer
from .spec import PartSpec


@register_mixer("side_by_side")
class SideBySide(Mixer):
    """left(h) + right(h), each a mixer of the registry with memory of its own (attention over pages beside a recurrence
    over a state, say); a factor on either result is its own ``out_scale``.

    Both give up their input projections (take_input()), which run as ONE product, and go on from its columns
    (forward_projected()); both results stay pending together (Product.also), so the next norm adds them.  In a step of
    few tokens the right mixer runs on a second stream beside the left one (in a captured graph: two branches).
    The left mixer's memory is the entry's own, the right one's is side memory "right".
    Parameters: left, right (PartSpecs).  Tensors: left.*, right.*.
    """

    #: up to this many tokens the two run side by side on two streams
    BRANCH_MAX_TOKENS = 64

    def __init__(self, spec: PartSpec, rt=None):
        super().__init__(spec, rt)
        self.left, self.right = MIXERS.build(spec["left"], rt=rt), MIXERS.build(spec["right"], rt=rt)
        for m in (self.left, self.right):
            if not hasattr(m, "forward_projected"):
                raise ValueError(f"a {m.spec.kind} mixer cannot share its input projection")
        self.weight = None
        self.col = 0

    def kernel_modules(self):
        return tuple(dict.fromkeys(self.left.kernel_modules() + self.right.kernel_modules()))

    def cache_need(self):
        return self.left.cache_need()

    def side_needs(self):
        out = {"left." + k: v for k, v in self.left.side_needs().items()}
        need = self.right.cache_need()
        if need is not None:
            out["right"] = need
        out.update({"right." + k: v for k, v in self.right.side_needs().items()})
        return out

    def side_user(self, name: str):
        if name == "right":
            return self.right
        side, _, rest = name.partition(".")
        return {"left": self.left, "right": self.right}[side].side_user(rest)

    def plan_key(self):
        return self.left.plan_key()

    def planner(self, page_size: int, sm_count: int):
        return self.left.planner(page_size, sm_count)

    def check_cache(self, page_size: int) -> None:
        self.left.check_cache(page_size)
        self.right.check_cache(page_size)

    @property
    def graph_safe(self) -> bool:
        return self.left.graph_safe and self.right.graph_safe

    def parameters(self):
        return {f"{side}.{k}": ps for side, m in (("left", self.left), ("right", self.right))
                for k, ps in m.parameters().items()}

    def load(self, tensors):
        for side, m in (("left", self.left), ("right", self.right)):
            m.load({k[len(side) + 1:]: t for k, t in tensors.items() if k.startswith(side + ".")})
        a, b = self.left.take_input(), self.right.take_input()
        self.col = a.shape[0]
        self.weight = _pad_rows(torch.cat((a, b), 0))

    def forward(self, h, ctx: StepContext, cache: CacheView) -> Product:
        left_view = cache.narrow("left.")
        right_view = cache.sides["right"].narrow("") if "right" in cache.sides else CacheView(None, -1, -1, True, None)
        right_view.sides = cache.narrow("right.").sides
        proj = ctx.rt.linear(h, self.weight, ctx.ws, "ab_proj", out_dtype=torch.float32)
        branch = ctx.extras.get("branch_stream") if h.shape[0] <= self.BRANCH_MAX_TOKENS else None
        if branch is None:
            a = self.left.forward_projected(proj, 0, ctx, left_view, "mix_out")
            b = self.right.forward_projected(proj, self.col, ctx, right_view, "mix_out_right")
            return Product(a.tensor, a.nsplit, also=b)
        # few tokens: two chains of small kernels that read the same product and write buffers of their own; their
        # products need no scratch shared between launches
        main = torch.cuda.current_stream()
        fork, join = ctx.extras["branch_events"]
        fork.record(main)
        branch.wait_event(fork)
        with torch.cuda.stream(branch), K.stream_scope():
            b = self.right.forward_projected(proj, self.col, ctx, right_view, "mix_out_right")
            join.record(branch)
        a = self.left.forward_projected(proj, 0, ctx, left_view, "mix_out")
        main.wait_event(join)
        return Product(a.tensor, a.nsplit, also=b)
