"""Zetenex on the host: the configuration reader, the spec it makes (repeated layers with a part that opens every pass),
the tensors it expects, the memory its layers ask for (pages, a state and kept inputs side by side), how the step function
hands it out, and the plain functions beside hand-made cases.  No GPU."""
import copy
import math

import pytest
import torch

from mini_hisparse_b200.cache import CacheConfig, CacheManager
from mini_hisparse_b200.config.qwen2 import ConfigError
from mini_hisparse_b200.config.registry import resolve
from mini_hisparse_b200.config.zetenex import ZetenexConfig
from mini_hisparse_b200.engine.step import BatchBuilder, StepEntry
from mini_hisparse_b200.parts.base import CacheView
from mini_hisparse_b200.parts.registry import BLOCKS
from mini_hisparse_b200.parts.spec import PagedKVNeed, StateNeed
from mini_hisparse_b200.weights.expected import expected_tensors_of_spec
from plain import zetenex_plain as P


def config():
    par = dict(left=dict(heads=4, kv_heads=2, dim=8, vdim=12, scale=0.3, q_temp=dict(coef=0.2, every=5)), left_scale=0.9,
               right=dict(inner=28, state=6, dt_rank=3, conv=3), right_scale=0.4)
    return dict(architecture="Zetenex", vocab=50, width=40, norm=dict(eps=1e-5), canon=dict(taps=5), embedding=dict(scale=2.5),
                layers=[dict(type="mingru", mixer=dict(width=36), mlp=dict(kind="dense", ff=24)),
                        dict(type="parallel", mixer=par, mlp=dict(kind="dense", ff=32)),
                        dict(type="mingru", mixer=dict(width=20), mlp=None)],
                loop=dict(start=1, stop=3, times=2))


def test_run_order_names_and_needs():
    cfg, spec = resolve(config())
    assert isinstance(cfg, ZetenexConfig) and cfg.taps == 5 and cfg.embedding_scale == 2.5
    assert [(e.layer, e.before, e.turn) for e in spec.order] == [(0, None, 0), (1, "loop", 0), (2, None, 0), (1, "loop", 1),
                                                                 (2, None, 1)]
    assert all(e.cache_of is None for e in spec.order)
    names = expected_tensors_of_spec(spec)
    shapes = {n: tuple(p.shape) for n, p in names.items() if not p.optional}
    norm = {f"{p}{s}": sh for p in ("l0.norm1", "l0.norm2", "l1.norm1", "l1.norm2", "l2.norm1", "final.norm")
            for s, sh in (("", (40,)), (".b", (40,)), (".alpha", ()))}
    assert shapes == {
        "embed": (50, 40), "loop.step": (2, 40), **norm,
        **{f"l{i}.canon{k}": (40, 5) for i, k in ((0, 1), (0, 2), (1, 1), (1, 2), (2, 1))},
        "l0.mix.z": (36, 40), "l0.mix.z.b": (36,), "l0.mix.x": (36, 40), "l0.mix.x.b": (36,), "l0.mix.g": (36, 40),
        "l0.mix.o": (40, 36), "l0.mlp.up": (24, 40), "l0.mlp.down": (40, 24),
        "l1.mix.left.q": (32, 40), "l1.mix.left.k": (16, 40), "l1.mix.left.v": (24, 40), "l1.mix.left.g": (4, 40),
        "l1.mix.left.o": (40, 48), "l1.mix.right.in": (56, 40), "l1.mix.right.conv": (28, 3), "l1.mix.right.conv.b": (28,),
        "l1.mix.right.x": (15, 28), "l1.mix.right.dt": (28, 3), "l1.mix.right.dt.b": (28,), "l1.mix.right.A_log": (28, 6),
        "l1.mix.right.D": (28,), "l1.mix.right.o": (40, 28), "l1.mlp.up": (32, 40), "l1.mlp.down": (40, 32),
        "l2.mix.z": (20, 40), "l2.mix.z.b": (20,), "l2.mix.x": (20, 40), "l2.mix.x.b": (20,), "l2.mix.g": (20, 40),
        "l2.mix.o": (40, 20)}
    blocks = [BLOCKS.get(layer.block)(layer, None) for layer in spec.layers]
    assert blocks[0].cache_need() == StateNeed(shape=(36,)) and blocks[0].side_needs() == {"input_conv": StateNeed(shape=(2, 4, 40))}
    assert blocks[1].cache_need() == PagedKVNeed(kv_heads=2, head_dim=8, v_dim=12)
    assert blocks[1].side_needs() == {"mixer.right": StateNeed(shape=(28 * 6 + 2 * 28,)), "input_conv": StateNeed(shape=(2, 4, 40))}
    assert blocks[2].side_needs() == {"input_conv": StateNeed(shape=(1, 4, 40))}          # no feed-forward, one convolution
    assert blocks[1].mixer.left.out_scale == 0.9 and blocks[1].mixer.right.out_scale == 0.4
    assert blocks[1].mixer.left.q_temp == (0.2, 5.0)


def test_side_memory_is_handed_out_by_name():
    """Entries with the same need share a group whether the memory is an entry's own or beside it; a view inside a view
    finds its part of the names."""
    _, spec = resolve(config())
    blocks = [BLOCKS.get(layer.block)(layer, None) for layer in spec.layers]
    needs, users = [], []
    for e in spec.order:
        b = blocks[e.layer]
        users.append((len(needs), {n: len(needs) + 1 + i for i, n in enumerate(b.side_needs())}, b))
        needs += [b.cache_need(), *b.side_needs().values()]
    cache = CacheManager(needs, CacheConfig(num_pages=6, page_size=4, max_requests=2, dtype=torch.float32, device="cpu"))
    batch = BatchBuilder(cache, "cpu", sm_count=8)
    main = [batch.add_user(at, b) for at, _, b in users]
    sides = [{n: batch.add_user(at, b.side_user(n)) for n, at in s.items()} for _, s, b in users]
    assert len(batch.slots) == 1                    # the attention's plan, shared by the layer's two runs
    cache.open("a")
    cache.ensure("a", 3)
    entries = [StepEntry("a", [1, 2, 3], [2])]
    segments, T = batch.segments(entries)
    views = batch.eager(entries, segments)
    assert views["seg_offset"].tolist() == [0, 3]
    seen = set()
    for i, m in enumerate(main):
        view = batch.cache_view(m, views)
        view.sides = {n: batch.cache_view(u, views) for n, u in sides[i].items()}
        for v in (view, *view.sides.values()):
            assert v.storage.data_ptr() not in seen             # every run entry has memory of its own
            seen.add(v.storage.data_ptr())
        if "mixer.right" in view.sides:
            inner = view.narrow("mixer.")
            assert set(inner.sides) == {"right"} and inner.storage is view.storage
            assert inner.sides["right"].storage.shape == (2, 28 * 8)
    assert isinstance(view, CacheView) and view.sides["input_conv"].storage.shape == (2, 1, 4, 40)
    # a slot that is used again starts from zero
    for g in cache.state_groups:
        g.storage.fill_(3.0)
    cache.close("a")
    slot = cache.open("b")
    assert all(float(g.storage[:, slot].abs().max()) == 0 for g in cache.state_groups)


def test_optional_pieces():
    c = config()
    del c["loop"], c["layers"][1]["mixer"]["left"]["q_temp"]
    cfg, spec = resolve(c)
    assert cfg.loop is None and not spec.shared and [e.layer for e in spec.order] == [0, 1, 2]
    assert "loop.step" not in expected_tensors_of_spec(spec)
    c["loop"] = None
    assert resolve(c)[0].loop is None
    c["loop"] = dict(start=0, stop=1, times=1)
    cfg, spec = resolve(c)
    assert [(e.layer, e.before) for e in spec.order] == [(0, "loop"), (1, None), (2, None)]
    c["canon"]["taps"] = 1                                       # nothing to keep
    _, spec = resolve(c)
    assert BLOCKS.get(spec.layers[0].block)(spec.layers[0], None).side_needs() == {}


@pytest.mark.parametrize("change,text", [
    (lambda c: c.update(extra=1), "unknown key"),
    (lambda c: c["layers"][1]["mixer"].update(mid=1), "unknown key"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(mask=dict(size=4)), "unknown key"),
    (lambda c: c["layers"][1]["mixer"]["left"]["q_temp"].update(floor=1), "unknown key"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not a feed-forward"),
    (lambda c: c["layers"][0].update(type="lstm"), "not a mixer"),
    (lambda c: c["layers"][1]["mixer"].pop("right_scale"), "lacks"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("conv"), "lacks"),
    (lambda c: c.pop("canon"), "lacks"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=3), "divisor"),
    (lambda c: c["layers"][1]["mixer"]["left"]["q_temp"].update(every=0), "positive"),
    (lambda c: c["loop"].update(stop=4), "make no sense"),
    (lambda c: c["loop"].update(stop=1), "make no sense"),
    (lambda c: c["loop"].update(times=0), "make no sense"),
    (lambda c: c["layers"][0]["mixer"].update(width=0), "positive"),
])
def test_what_the_reader_refuses(change, text):
    c = copy.deepcopy(config())
    change(c)
    with pytest.raises(ConfigError, match=text):
        ZetenexConfig.from_dict(c)


def test_plain_functions_by_hand():
    h = torch.tensor([[1.0], [2.0], [3.0], [4.0]], dtype=torch.float64)
    y = P.with_convolution(h, torch.tensor([[100.0, 10.0, 1.0]], dtype=torch.float64))       # the last tap is the current token's
    assert y[:, 0].tolist() == [2.0, 14.0, 126.0, 238.0]
    # the temperature steps when (p + 1) reaches a multiple of every
    t = P.query_temperature([0, 3, 4, 5, 9], dict(coef=0.5, every=5))
    assert t.tolist() == pytest.approx([1, 1, 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(2), 1 + 0.5 * math.log(3)])
    # minGRU: a gate that is open takes the candidate, one that is shut keeps the state; both branches of the candidate
    zl = torch.tensor([[40.0], [-40.0], [40.0], [0.0]], dtype=torch.float64)
    u = torch.tensor([[2.0], [9.0], [-1.0], [0.0]], dtype=torch.float64)
    S = P.gru_states(zl, u)[:, 0].tolist()
    low = 1 / (1 + math.e)
    assert S == pytest.approx([2.5, 2.5, low, 0.5 * low + 0.25])
    # the scan: one channel, one state, decay exp(-1) a step
    one = torch.ones(3, 1, dtype=torch.float64)
    y, last = P.selective_states(one * 2.0, one, -one[:1], one * 3.0, one)
    assert y[:, 0].tolist() == pytest.approx([6.0, 6 + 6 * math.exp(-1), 6 + 6 * math.exp(-1) + 6 * math.exp(-2)])
    assert float(last[0, 0]) == pytest.approx(float(y[2, 0]))
    # attention: every earlier key and the token's own
    k = torch.zeros(4, 1, 2, dtype=torch.float64)
    v = torch.arange(4, dtype=torch.float64).view(4, 1, 1)
    assert P.causal_softmax(torch.zeros(4, 2, 2, dtype=torch.float64), k, v, 1.0)[:, 1, 0].tolist() == pytest.approx([0, 0.5, 1.0, 1.5])
