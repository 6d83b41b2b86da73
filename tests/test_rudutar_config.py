"""Rudutar on the host: the configuration reader and what it refuses, the spec it makes (a layer that reads another
layer's keys, a layer without a feed-forward), the tensors it expects, the memory its layers ask for, and the plain
functions beside hand-made cases.  No GPU."""
import copy
import math

import pytest
import torch

from mini_hisparse_b200.config.qwen2 import ConfigError
from mini_hisparse_b200.config.registry import resolve
from mini_hisparse_b200.config.rudutar import RudutarConfig
from mini_hisparse_b200.parts.registry import BLOCKS, FEED_FORWARDS, MIXERS
from mini_hisparse_b200.parts.spec import PagedKVNeed, PartSpec, StateNeed
from mini_hisparse_b200.weights.expected import expected_tensors_of_spec
from plain import rudutar_plain as P


def config():
    att = dict(heads=6, kv_heads=3, dim=8, vdim=12, conv=4, scale=0.4, mask=dict(size=9), q_temp=dict(coef=0.2, every=7))
    key = dict(heads=4, kv_heads=2, dim=10, vdim=10, scale=0.3, mask=dict(size=5), rot=dict(dims=6, base=50.0))
    moe = dict(kind="moe", expert=dict(ff=24), shared=dict(ff=40),
               router=dict(experts=8, top=2, scale=2.5, groups=dict(count=4, keep=2)))
    return dict(architecture="Rudutar", vocab=50, width=40, norm=dict(eps=1e-5), layers=[
        dict(type="attention", mixer=dict(att), mlp=dict(kind="dense", ff=48)),
        dict(type="attention_2", mixer=dict(key), mlp=moe),
        dict(type="attention", mixer=dict(att, kv_from=0, heads=3, mask=dict(size=21)), mlp=None),
        dict(type="attention", mixer=dict(att, conv=1), mlp=dict(kind="dense", ff=8))])


def test_run_order_names_and_cache_needs():
    cfg, spec = resolve(config())
    assert isinstance(cfg, RudutarConfig) and cfg.layers[1].mlp.scale == 2.5
    assert [(e.layer, e.cache_of) for e in spec.order] == [(0, None), (1, None), (2, 0), (3, None)]
    names = {n: ps.shape for n, ps in expected_tensors_of_spec(spec).items()}
    want = {"embed": (50, 40), "embed.norm": (40,), "final.norm": (40,), "head": (50, 40)}
    for i, (q, conv) in {0: (48, 4), 2: (24, 4), 3: (48, 1)}.items():
        want.update({f"l{i}.norm1": (40,), f"l{i}.mix.q": (q, 40), f"l{i}.mix.q.norm": (8,), f"l{i}.mix.q.conv": (q, conv),
                     f"l{i}.mix.g": (q // 8 * 12, 40), f"l{i}.mix.o": (40, q // 8 * 12)})
        if i != 2:
            want.update({f"l{i}.mix.k": (24, 40), f"l{i}.mix.v": (36, 40), f"l{i}.mix.k.norm": (8,),
                         f"l{i}.mix.k.conv": (24, conv), f"l{i}.mix.v.conv": (36, conv), f"l{i}.norm2": (40,)})
    want.update({"l0.mlp.up": (48, 40), "l0.mlp.down": (40, 48), "l3.mlp.up": (8, 40), "l3.mlp.down": (40, 8)})
    want.update({"l1.norm1": (40,), "l1.norm2": (40,), "l1.mix.q": (40, 40), "l1.mix.q.b": (40,), "l1.mix.k": (20, 40),
                 "l1.mix.k.b": (20,), "l1.mix.q.norm": (40,), "l1.mix.k.norm": (20,), "l1.mix.g": (4, 40),
                 "l1.mix.o": (40, 40), "l1.mlp.router": (8, 40), "l1.mlp.correction": (8,), "l1.mlp.shared.up": (40, 40),
                 "l1.mlp.shared.down": (40, 40)})
    for e in range(8):
        want.update({f"l1.mlp.e{e}.up": (24, 40), f"l1.mlp.e{e}.down": (40, 24)})
    assert names == want
    # the first layer's pages live as long as the widest window of its readers; its own queries see 9 positions
    mixers = [MIXERS.build(layer.part("mixer")) for layer in spec.layers]
    assert mixers[0].cache_need() == PagedKVNeed(kv_heads=3, head_dim=8, window=21, v_dim=12) == mixers[2].cache_need()
    assert (mixers[0].window, mixers[2].window) == (9, 21) and mixers[0].own_kv and not mixers[2].own_kv
    assert mixers[1].cache_need() == PagedKVNeed(kv_heads=2, head_dim=10, window=5)
    assert mixers[3].cache_need() == PagedKVNeed(kv_heads=3, head_dim=8, window=9, v_dim=12)
    # kept rows of the convolutions: q, k and v; q alone for the reader; none for a single tap
    blocks = [BLOCKS.get(layer.block)(layer, None) for layer in spec.layers]
    assert [b.side_needs() for b in blocks] == [{"mixer.conv": StateNeed(shape=(3, 48 + 24 + 36))}, {},
                                                {"mixer.conv": StateNeed(shape=(3, 24))}, {}]
    assert sorted(blocks[2].parts()) == ["mixer", "mixer_norm"]


def test_what_may_be_left_out():
    c = config()
    c["layers"][0]["mixer"].pop("q_temp")
    c["layers"][1]["mixer"].pop("rot")
    c["layers"][1]["mlp"].pop("shared")
    c["layers"][1]["mlp"]["router"].pop("groups")
    c["layers"][1]["mlp"]["router"].pop("scale")
    cfg, spec = resolve(c)
    assert cfg.layers[0].mixer.q_temp is None and cfg.layers[1].mixer.rot_dims == 0
    assert (cfg.layers[1].mlp.group_count, cfg.layers[1].mlp.group_keep, cfg.layers[1].mlp.scale) == (1, 1, 1.0)
    assert not any("shared" in n for n in expected_tensors_of_spec(spec))


def test_what_the_reader_refuses():
    def router(c):
        return c["layers"][1]["mlp"]["router"]

    for change in (lambda c: c.update(extra=1), lambda c: c.pop("width"), lambda c: c["norm"].update(kind="rms"),
                   lambda c: c.update(layers=[]), lambda c: c["layers"][0].update(type="latent"),
                   lambda c: c["layers"][0].update(weights_of=1), lambda c: c["layers"][0]["mixer"].pop("conv"),
                   lambda c: c["layers"][0]["mixer"].update(conv=17), lambda c: c["layers"][0]["mixer"].update(sink=1.0),
                   lambda c: c["layers"][0]["mixer"].update(rot=dict(dims=2, base=10.0)),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(chunk=8), lambda c: c["layers"][0]["mixer"].pop("mask"),
                   lambda c: c["layers"][0]["mixer"]["q_temp"].update(every=0),
                   lambda c: c["layers"][0]["mixer"].update(kv_heads=4), lambda c: c["layers"][1]["mixer"].update(vdim=12),
                   lambda c: c["layers"][1]["mixer"].update(conv=2), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=5),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=12),
                   lambda c: c["layers"][2]["mixer"].update(kv_from=1), lambda c: c["layers"][2]["mixer"].update(kv_from=2),
                   lambda c: c["layers"][2]["mixer"].update(kv_from=3), lambda c: c["layers"][2]["mixer"].update(vdim=16),
                   lambda c: c["layers"][3]["mixer"].update(kv_from=2),              # which has no keys of its own
                   lambda c: c["layers"][0]["mlp"].update(kind="routed"), lambda c: c["layers"][0]["mlp"].pop("ff"),
                   lambda c: router(c).update(top=5), lambda c: router(c)["groups"].update(count=3),
                   lambda c: router(c)["groups"].update(keep=5), lambda c: router(c).update(identity=1),
                   lambda c: c["layers"][1]["mlp"]["shared"].update(kind="dense")):
        c = copy.deepcopy(config())
        change(c)
        with pytest.raises(ConfigError):
            RudutarConfig.from_dict(c)


def test_parts_refuse_what_they_cannot_compute():
    base = dict(hidden_size=32, q_heads=2, kv_heads=1, dim=8, vdim=8, scale=0.3, window=4, eps=1e-5)
    with pytest.raises(ValueError, match="does not rotate"):
        MIXERS.build(PartSpec.make("sloped_attention", conv=2, position=PartSpec.make("rotary", head_dim=8, theta=10.0), **base))
    with pytest.raises(ValueError, match="owns its cache"):
        MIXERS.build(PartSpec.make("key_value_attention", position=PartSpec.make("none"), own_kv=False, **base))
    with pytest.raises(ValueError, match="as wide as"):
        MIXERS.build(PartSpec.make("key_value_attention", position=PartSpec.make("none"), **dict(base, vdim=12)))
    with pytest.raises(ValueError, match="form"):
        FEED_FORWARDS.build(PartSpec.make("routed_experts", hidden_size=32, experts=4, top=1, expert_ff=8, form="tanh"))
    with pytest.raises(ValueError, match="scores"):
        FEED_FORWARDS.build(PartSpec.make("routed_experts", hidden_size=32, experts=4, top=1, expert_ff=8, score="relu"))


# ---- the plain functions beside cases made by hand -------------------------------------------------------------
def test_the_plain_router_on_a_case_made_by_hand():
    """Six outputs in three groups of which two are kept.  Group (0, 1) has the largest single score but the smallest sum;
    every choice score is negative, so a dropped group must not win by counting as zero; weights carry no correction."""
    s = torch.tensor([0.9, 0.02, 0.6, 0.55, 0.5, 0.45], dtype=torch.float64)
    w = {"router": torch.eye(6, dtype=torch.float64), "correction": torch.full((6,), -2.0, dtype=torch.float64)}
    h = torch.log(s / (1 - s))[None]
    chosen, weights = P.route(h, w, "", dict(top=3, scale=1.5, groups=dict(count=3, keep=2)))
    assert chosen[0].tolist() == [2, 3, 4]
    torch.testing.assert_close(weights[0], 1.5 * s[2:5])
    chosen, weights = P.route(h, w, "", dict(top=3, scale=1.0, groups=None))
    assert chosen[0].tolist() == [0, 2, 3]
    w["correction"][5] = -1.0                      # lifts group (4, 5), and 5 in it
    chosen, weights = P.route(h, w, "", dict(top=2, scale=1.0, groups=dict(count=3, keep=1)))
    assert chosen[0].tolist() == [5, 4]
    torch.testing.assert_close(weights[0], s[[5, 4]])
    chosen, _ = P.route(h, w, "", dict(top=1, groups=dict(count=6, keep=1)))         # groups of one: no second score
    assert chosen[0].tolist() == [5]


def test_the_plain_attention_on_cases_made_by_hand():
    # one head, three positions, a window of two, slope 2^-8: by hand
    q, k = torch.tensor([1.0, 2.0, 3.0]).double().view(3, 1, 1), torch.tensor([1.0, -1.0, 0.5]).double().view(3, 1, 1)
    v = torch.tensor([10.0, 20.0, 30.0]).double().view(3, 1, 1)
    out = P.window_attend(q, k, v, 0.5, 2, slope=P.slopes(1), sink=True).flatten()
    a, b = math.exp(3 * -1.0 * 0.5 - 1 / 256), math.exp(3 * 0.5 * 0.5)
    assert abs(float(out[2]) - (20 * a + 30 * b) / (1 + a + b)) < 1e-12
    assert abs(float(out[0]) - 10 * math.exp(0.5) / (1 + math.exp(0.5))) < 1e-12
    plain = P.window_attend(q, k, v, 0.5, 1).flatten()            # a window of one: the token itself
    torch.testing.assert_close(plain, v.flatten())
    assert [float(x) for x in P.slopes(4)] == [2.0 ** -2, 2.0 ** -4, 2.0 ** -6, 2.0 ** -8]
    t = P.temperature(torch.tensor([0, 5, 6, 13, 12]), 0.2, 7)
    torch.testing.assert_close(t, torch.tensor([1.0, 1.0, 1 + 0.2 * math.log(2), 1 + 0.2 * math.log(3), 1 + 0.2 * math.log(2)]).double())
    y = P.short_convolution(torch.tensor([[1.0], [2.0], [4.0]]).double(), torch.tensor([[0.5, 3.0]]).double())
    assert y.flatten().tolist() == [3.0, 6.5, 13.0]
    assert abs(float(P.gelu(torch.tensor(1.0).double())) - 0.8413447460685429) < 1e-12
