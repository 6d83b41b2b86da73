"""Zetenex through the engine against the plain implementation of tests/plain/zetenex_plain.py.

Small configurations made here (none is anyone's model), random weights from a seed.  Covered: the kernels of each
mechanism alone (the norm with the convolution behind it over segments that start, go on and end anywhere, with the kept
inputs; the convolution of a product's columns; the chosen rows' norm; the opening of a pass; minGRU token by token and in
runs; the selective scan for few and many states, channels and tokens, from a slot's state and from zero; unit q and k with
the temperature at its steps; the gelu in the product's epilogue); the two mixers alone over hand-made inputs in which one
key far back stands out, and one write that has to be remembered; whole prompts; prefill against token-by-token decoding
through captured graphs; portions down to two tokens; mixed batches over a tight pool whose freed pages are poisoned; slots
used again; long decoding; sizes that are equal or 1; generation through Engine and its scheduler; the command line;
bin/trace_run.
"""
import copy
import json

import pytest
import torch

import schedules as S
from conftest import TraceRun, random_tokens, row_rms_error
from plain import zetenex_plain as P
from test_dotivik_gpu import Parts, dev_i, run_steps

pytestmark = pytest.mark.gpu


def left(heads, kv_heads, dim, vdim, scale=0.3, temp=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale)
    if temp is not None:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    return m


def right(inner, state, dt_rank, conv):
    return dict(inner=inner, state=state, dt_rank=dt_rank, conv=conv)


def parallel(a, b, ff=None, scales=(0.8, 0.6)):
    return dict(type="parallel", mixer=dict(left=a, right=b, left_scale=scales[0], right_scale=scales[1]),
                mlp=None if ff is None else dict(kind="dense", ff=ff))


def gru(width, ff=None):
    return dict(type="mingru", mixer=dict(width=width), mlp=None if ff is None else dict(kind="dense", ff=ff))


def model(vocab, width, layers, taps=4, loop=None, scale=3.0, eps=1e-5):
    cfg = dict(architecture="Zetenex", vocab=vocab, width=width, norm=dict(eps=eps), canon=dict(taps=taps),
               embedding=dict(scale=scale), layers=layers)
    if loop is not None:
        cfg["loop"] = dict(start=loop[0], stop=loop[1], times=loop[2])
    return cfg


# A: every branch at once: both mixers with and without a feed-forward, keys narrower than values, a temperature that steps
# many times within a prompt, a loop that starts at the first layer.
CFG_A = model(211, 88, [parallel(left(6, 3, 24, 40, temp=(0.4, 7)), right(72, 12, 6, 3), ff=120), gru(104, ff=72), gru(56),
                        parallel(left(4, 1, 32, 16, scale=0.5), right(40, 20, 10, 5)), gru(64, ff=40)], taps=3, loop=(0, 3, 2))
# B: values that a usual model makes different are equal or 1 here: one head, one state, a step of rank one, filters of one
# tap, a pass that runs once, factors of one, a width that no tensor-core product takes, pages of eight.
CFG_B = model(97, 100, [gru(1, ff=4), parallel(left(1, 1, 20, 20, temp=(1.0, 1)), right(20, 1, 1, 1), ff=20, scales=(1.0, 1.0)),
                        parallel(left(5, 5, 12, 8), right(100, 3, 9, 2), scales=(0.0, 1.5)), gru(100)], taps=1,
              loop=(2, 3, 1), scale=1.0, eps=1e-3)
# C: sizes of a real model's order: heads of 64 that the tcgen05 tiles take, sixteen states, a loop of one layer in the
# middle; pages of 32.
CFG_C = model(300, 256, [gru(320, ff=512), parallel(left(8, 2, 64, 64, scale=0.2, temp=(0.1, 50)), right(256, 16, 16, 4), ff=512),
                         gru(256, ff=384)], loop=(1, 2, 3), scale=8.0)
# D: long filters (the scalar path of the convolution kernels), many states a channel, heads of 128.
CFG_D = model(150, 136, [parallel(left(3, 1, 128, 128, scale=0.1), right(48, 70, 8, 7), ff=64),
                         parallel(left(2, 2, 16, 24, temp=(0.3, 30)), right(24, 140, 24, 16)), gru(40, ff=48)], taps=9, scale=2.0)
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C, "D": CFG_D}
PAGES = {"A": 16, "B": 8, "C": 32, "D": 16}
# The matrices' standard deviation: the scan's output is a product of three projections of its input and nothing bounds it,
# so with wide layers and large matrices the stream grows until even float32 and float64 runs of one program part.
STD = {"A": 0.15, "B": 0.15, "C": 0.08, "D": 0.12}
# A row's error: the root mean square of (got - plain) as a share of the row's root mean square.  The plain model is
# computed in float64.  bfloat16: activations are rounded to 8 bits after every part of up to nine layer runs.
F32_ROW, BF16_ROW, BF16_MEAN = 3e-5, 0.09, 0.03


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    from mini_hisparse_b200 import write_random_model

    out = {}
    for name, cfg in CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"zetenex{name}")
        write_random_model(cfg, 53, folder, dtype=torch.bfloat16, matrix_std=STD[name])
        out[name] = (folder, *P.load_folder(folder))
    return out


def requests_for(cfg, lengths, seed=0):
    return {f"r{i}": random_tokens(cfg["vocab"], n, seed + i) for i, n in enumerate(lengths)}


def row_errors(got, ref):
    return (got.double() - ref.double()).pow(2).mean(-1).sqrt() / ref.double().pow(2).mean(-1).sqrt()


def check_rows(err, dtype):
    worst, mean = float(err.max()), float(err.mean())
    if dtype == "float32":
        assert worst < F32_ROW, f"worst row error {worst:.3g} at {int(err.argmax())}"
    else:
        assert worst < BF16_ROW and mean < BF16_MEAN, f"worst row error {worst:.3g} at {int(err.argmax())}, mean {mean:.3g}"


def check_against_plain(got, refs, dtype):
    for rid, ref in refs.items():
        assert got[rid].shape == ref.shape
    check_rows(torch.cat([row_errors(got[rid], ref) for rid, ref in refs.items()]), dtype)


def close(got, ref, tol, what=""):
    ref = ref.double()
    err = float((got.double().cpu() - ref).abs().max())
    assert err <= tol * max(1.0, float(ref.abs().max())), f"{what}: off by {err:.3g}"


class Batch:
    """A step's segments as the kernels' wrappers read them: counts, first positions and slots."""

    def __init__(self, counts, starts, slots):
        self.counts, self.starts, self.slots = counts, starts, slots
        self.T = sum(counts)
        self.offsets = [sum(counts[:i]) for i in range(len(counts) + 1)]
        self.seg_offset, self.seg_slot = dev_i(self.offsets), dev_i(slots)
        self.positions = dev_i([s + i for s, n in zip(starts, counts) for i in range(n)])
        self.segments, self.longest = counts, max(counts)

    def rows(self, i):
        return slice(self.offsets[i], self.offsets[i + 1])


# segments that start a sequence, go on after few or many tokens, hold one token, fewer than a filter's taps, exactly a
# tile of the convolution kernel, one more, and several tiles; slots in no order
BATCHES = [([1, 2, 5, 16, 17, 40, 3], [0, 9, 0, 4, 0, 1, 2], [5, 0, 3, 6, 1, 2, 4]), ([1, 1, 1], [0, 7, 1], [2, 0, 1]),
           ([70], [0], [0]), ([33], [50], [1])]


# ---- the kernels of each mechanism alone --------------------------------------------------------------------
@pytest.mark.parametrize("C,taps", [(96, 4), (100, 3), (33, 2), (64, 1), (40, 6), (24, 16)])
@pytest.mark.parametrize("batch", range(len(BATCHES)))
def test_norm_and_convolution_in_one_kernel(C, taps, batch):
    from mini_hisparse_b200.kernels import api as K

    b = Batch(*BATCHES[batch])
    g = torch.Generator().manual_seed(C + taps)
    x, d1, d2 = torch.randn(b.T, C, generator=g), torch.randn(3, b.T, C, generator=g), torch.randn(b.T, C, generator=g)
    f, w, shift = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(C, generator=g)
    alpha = torch.tensor([0.7])
    keep = torch.randn(7, 2, max(taps - 1, 1), C, generator=g)
    for out_dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 1e-2)):
        for deltas in (0, 1, 2):
            total = x.double() + (d1.double().sum(0) if deltas else 0) + (d2.double() if deltas == 2 else 0)
            h = P.dynamic_tanh(total, alpha.double(), w.double(), shift.double())
            kept, out = keep.cuda(), torch.empty(b.T, C, dtype=out_dtype, device="cuda")
            x_out = torch.full((b.T, C), 7.0, device="cuda")
            K.stream_conv(x.cuda(), alpha.cuda(), w.cuda(), shift.cuda(), f.t().contiguous().cuda(), kept[:, 1] if taps > 1 else None, b,
                          out, delta=Parts(d1.cuda(), 3) if deltas else None, delta2=Parts(d2.cuda()) if deltas == 2 else None,
                          x_out=x_out if deltas else None)
            if deltas:
                close(x_out, total, 3e-6, "the sum")
            for i, (n, start, slot) in enumerate(zip(b.counts, b.starts, b.slots)):
                before = keep[slot, 1].double()[:taps - 1] if start else torch.zeros(taps - 1, C).double()
                # (a slot that goes on holds what a test wrote there, also at places before the sequence's start)
                both = torch.cat((before, h[b.rows(i)]), 0)
                ref = P.with_convolution(both, f.double())[taps - 1:]
                close(out[b.rows(i)], ref, tol, f"segment {i}")
                if taps > 1:
                    close(kept[slot, 1, :taps - 1], both[n:], 3e-6, f"kept inputs of segment {i}")
            assert torch.equal(kept[:, 0].cpu(), keep[:, 0])               # the other convolution's inputs
            untouched = [s for s in range(7) if s not in b.slots]
            assert torch.equal(kept[untouched].cpu(), keep[untouched])
    # behind another norm: rows as they are
    for dtype, tol in ((torch.float32, 3e-6), (torch.bfloat16, 1e-2)):
        hd, kept = x.to(dtype), keep.cuda()
        out = torch.empty(b.T, C, dtype=dtype, device="cuda")
        K.rows_conv(hd.cuda(), f.t().contiguous().cuda(), kept[:, 1] if taps > 1 else None, b, out)
        for i, (n, start, slot) in enumerate(zip(b.counts, b.starts, b.slots)):
            before = keep[slot, 1].double()[:taps - 1] if start else torch.zeros(taps - 1, C).double()
            both = torch.cat((before, hd[b.rows(i)].double()), 0)
            close(out[b.rows(i)], P.with_convolution(both, f.double())[taps - 1:], tol, f"rows, segment {i}")
            if taps > 1:
                close(kept[slot, 1, :taps - 1], both[n:], 0, f"rows, kept inputs of segment {i}")


@pytest.mark.parametrize("C,taps,nsplit,c0", [(96, 4, 1, 16), (96, 4, 3, 3), (20, 1, 2, 0), (36, 2, 1, 8), (24, 7, 2, 4)])
@pytest.mark.parametrize("batch", range(len(BATCHES)))
def test_convolution_of_a_products_columns(C, taps, nsplit, c0, batch):
    from mini_hisparse_b200.kernels import api as K

    b = Batch(*BATCHES[batch])
    g = torch.Generator().manual_seed(C + taps)
    proj = torch.randn(nsplit, b.T, c0 + C + 8, generator=g)
    f, bias, keep = torch.randn(C, taps, generator=g), torch.randn(C, generator=g), torch.randn(7, 5 + (taps - 1) * C, generator=g)
    z = proj.double().sum(0)[:, c0:c0 + C]
    kept, out, out32 = keep.cuda(), torch.empty(b.T, C, dtype=torch.bfloat16, device="cuda"), torch.empty(b.T, C, device="cuda")
    K.product_conv(Parts(proj.cuda() if nsplit > 1 else proj[0].cuda(), nsplit), c0, f.t().contiguous().cuda(), bias.cuda(),
                   kept[:, 5:] if taps > 1 else None, b, out, out32=out32)
    for i, (n, start, slot) in enumerate(zip(b.counts, b.starts, b.slots)):
        before = keep[slot, 5:].double().view(taps - 1, C) if start else torch.zeros(taps - 1, C).double()
        both = torch.cat((before, z[b.rows(i)]), 0)
        ref = P.silu(P.convolve(both, f.double())[taps - 1:] + bias.double())
        close(out32[b.rows(i)], ref, 3e-6, f"segment {i}")
        close(out[b.rows(i)], ref, 1e-2, f"segment {i}, rounded")
        if taps > 1:
            close(kept[slot, 5:].view(taps - 1, C), both[n:], 1e-6, f"kept inputs of segment {i}")
    assert torch.equal(kept[:, :5].cpu(), keep[:, :5])


@pytest.mark.parametrize("H", [96, 33, 1100])
def test_rows_norm_and_the_opening_of_a_pass(H):
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(H)
    T = 9
    x, d1, d2 = torch.randn(T, H, generator=g), torch.randn(2, T, H, generator=g), torch.randn(T, H, generator=g)
    w, shift, row, alpha = torch.randn(H, generator=g), torch.randn(H, generator=g), torch.randn(H, generator=g), torch.tensor([1.3])
    total = x.double() + d1.double().sum(0) + d2.double()
    rows = torch.tensor([8, 0, 3, 3])
    xd, out = x.cuda(), torch.empty(4, H, device="cuda")
    K.dyt_rows(xd, alpha.cuda(), w.cuda(), shift.cuda(), out, delta=Parts(d1.cuda(), 2), delta2=Parts(d2.cuda()), rows=dev_i(rows))
    close(out, P.dynamic_tanh(total[rows], 1.3, w.double(), shift.double()), 3e-6)
    assert torch.equal(xd.cpu(), x)                                    # chosen rows only: the stream stays as it is
    out = torch.empty(T, H, dtype=torch.bfloat16, device="cuda")
    K.dyt_rows(xd, alpha.cuda(), w.cuda(), shift.cuda(), out, delta=Parts(d1.cuda(), 2))
    close(xd, x.double() + d1.double().sum(0), 3e-6)
    close(out, P.dynamic_tanh(x.double() + d1.double().sum(0), 1.3, w.double(), shift.double()), 1e-2)
    # the opening of a pass
    tokens, scale = torch.randint(0, 20, (T,), generator=g), 2.5
    for table_dtype in (torch.float32, torch.bfloat16):
        table = torch.randn(20, H, generator=g).to(table_dtype)
        for with_delta in (False, True):
            for with_table in (False, True):
                xd = x.cuda()
                K.stream_shift(xd, row.cuda(), delta=Parts(d1.cuda(), 2) if with_delta else None,
                               table=table.cuda() if with_table else None, tokens=dev_i(tokens), scale=scale)
                ref = x.double() + row.double() + (d1.double().sum(0) if with_delta else 0)
                close(xd, ref + (table.double()[tokens] * scale if with_table else 0), 3e-6)


@pytest.mark.parametrize("W,nsplit", [(96, 1), (20, 3), (1, 2), (333, 1)])
@pytest.mark.parametrize("counts,starts,slots", [([1, 3, 16, 2], [0, 5, 0, 40], [2, 0, 3, 1]), ([1, 17, 600, 5], [3, 0, 9, 0], [1, 3, 0, 2]),
                                                 ([1100], [0], [0]), ([512, 513], [0, 6], [1, 0])])
def test_mingru_recurrence(W, nsplit, counts, starts, slots):
    """Short segments token by token, long ones in runs; the state of a slot is taken up and left behind."""
    from mini_hisparse_b200.kernels import api as K

    b = Batch(counts, starts, slots)
    g = torch.Generator().manual_seed(W)
    z0, x0, g0 = 4, 4 + W, 9 + 2 * W
    proj = torch.randn(nsplit, b.T, g0 + W + 3, generator=g)
    proj[0, :, z0:z0 + W] -= 3.0                              # gates that are mostly shut: the state reaches far back
    bz, bx, state = torch.randn(W, generator=g), torch.randn(W, generator=g), torch.randn(4, W + 6, generator=g)
    p = proj.double().sum(0)
    for out_dtype, tol in ((torch.float32, 2e-5), (torch.bfloat16, 1e-2)):
        sd, out = state.cuda(), torch.empty(b.T, W, dtype=out_dtype, device="cuda")
        K.mingru_scan(Parts(proj.cuda() if nsplit > 1 else proj[0].cuda(), nsplit), z0, x0, g0, bz.cuda(), bx.cuda(), sd, b, out)
        for i, (n, start, slot) in enumerate(zip(counts, starts, slots)):
            r = p[b.rows(i)]
            ref = P.gru_states(r[:, z0:z0 + W] + bz, r[:, x0:x0 + W] + bx, state[slot, :W].double() if start else None)
            close(out[b.rows(i)], ref * P.silu(r[:, g0:g0 + W]), tol, f"segment {i}")
            close(sd[slot, :W], ref[-1], 2e-5, f"state after segment {i}")
        assert torch.equal(sd[:, W:].cpu(), state[:, W:])


@pytest.mark.parametrize("C,N,R,nsplit", [(80, 12, 6, 1), (20, 1, 1, 2), (33, 16, 16, 3), (560, 16, 24, 1), (48, 24, 8, 1), (600, 20, 8, 1),
                                          (560, 32, 9, 2), (40, 33, 5, 1), (24, 70, 8, 1), (24, 140, 24, 1), (10, 256, 3, 1)])
def test_selective_scan(C, N, R, nsplit):
    """Few tokens (the step's product inside) and many (walking and helping warps), fresh slots and slots that go on;
    decays from nearly none to nearly all."""
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(C + N)
    A = -torch.exp(torch.linspace(-6, 2, C * N)[torch.randperm(C * N, generator=g)].view(C, N))
    A2 = (A * 1.4426950408889634).contiguous()
    D, bias = torch.randn(C, generator=g), torch.randn(C, generator=g) - 1.0
    Wdt = (torch.randn(C, R, generator=g) / R ** 0.5).to(torch.bfloat16)
    state = torch.randn(7, C * N + 5, generator=g)
    cases = [Batch([1, 3, 16, 2], [0, 5, 0, 40], [2, 0, 3, 1]), Batch([1, 1], [8, 0], [4, 1]),
             Batch([40, 1, 17, 75, 2, 5, 32], [0, 5, 9, 3, 0, 77, 0], [2, 0, 3, 1, 6, 4, 5]), Batch([130], [0], [6])]
    for ci, b in enumerate(cases):
        low = torch.randn(nsplit, b.T, R + 2 * N + 3, generator=g)
        proj = torch.randn(2, b.T, 2 * C + 4, generator=g)
        x = torch.randn(b.T, C, generator=g)
        ls, zs = low.double().sum(0), proj.double().sum(0)[:, C:2 * C]
        lp = Parts(low.cuda() if nsplit > 1 else low[0].cuda(), nsplit)
        pp = Parts(proj.cuda(), 2)
        for dtype in (torch.float32, torch.bfloat16):
            W = Wdt.to(dtype)
            out, sd = torch.empty(b.T, C, dtype=dtype, device="cuda"), state.cuda()
            args = (A2.cuda(), D.cuda(), sd, b, out)
            if ci < 2:
                K.selective_scan(pp, C, lp, lp, R, x.cuda(), bias.cuda(), *args, dt_weight=W.cuda(), rank=R, scale=0.7)
                logits = ls[:, :R] @ Wdt.double().T
            else:
                pad = -(-R // 8) * 8
                dt_in, bc = torch.empty(b.T, pad, dtype=dtype, device="cuda"), torch.empty(b.T, 2 * N, device="cuda")
                K.selective_split(lp, R, N, dt_in, bc)
                close(dt_in[:, :R], ls[:, :R], 3e-6 if dtype == torch.float32 else 1e-2, "the step's columns")
                assert float(dt_in[:, R:].float().abs().sum()) == 0
                close(bc, ls[:, R:R + 2 * N], 3e-6, "B and C")
                logits = dt_in[:, :R].double().cpu() @ Wdt.double().T
                K.selective_scan(pp, C, Parts(logits.float().cuda()), Parts(bc), 0, x.cuda(), bias.cuda(), *args, scale=0.7)
            dt = P.softplus(logits + bias.double())
            for i, (n, start, slot) in enumerate(zip(b.counts, b.starts, b.slots)):
                r = b.rows(i)
                y, last = P.selective_states(x[r].double(), dt[r], A.double(), ls[r, R:R + N], ls[r, R + N:R + 2 * N],
                                             state[slot, :C * N].double().view(C, N) if start else None)
                ref = (y + D.double() * x[r].double()) * P.silu(zs[r]) * 0.7
                close(out[r], ref, 2e-5 if dtype == torch.float32 else 1e-2, f"case {ci}, segment {i}")
                close(sd[slot, :C * N].view(C, N), last, 2e-5, f"case {ci}, state after segment {i}")
            assert torch.equal(sd[:, C * N:].cpu(), state[:, C * N:])


@pytest.mark.parametrize("nq,nkv,dk,dv,P_,temp", [(6, 3, 24, 40, 16, (0.4, 7)), (1, 1, 20, 20, 8, None), (4, 2, 64, 64, 16, (1.0, 1)),
                                                  (4, 2, 64, 64, 16, (0.25, 2.5))])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unit_queries_and_keys_with_a_temperature(nq, nkv, dk, dv, P_, temp, dtype):
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(nq)
    positions = [0, 1, 4, 5, 6, 7, 12, 13, 14, 48, 49, 95]             # around the steps of the temperature
    T, wide = len(positions), nq * dk + nkv * (dk + dv)
    proj = torch.randn(2, T, 5 + wide + nq, generator=g)
    p = proj.double().sum(0)[:, 5:]
    cache = torch.zeros(13, nkv * P_ * (dk + dv), dtype=dtype, device="cuda")
    pages = torch.randperm(13, generator=g)[:96 // P_]
    q = torch.empty(T, nq * dk, dtype=dtype, device="cuda")
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    K.qknorm_rope_append(proj.cuda()[..., 5:], None, None, 1e-4, dev_i(positions), dev_i([0] * T), dev_i(pages[None]), None, 0, q, cache,
                         nq=nq, nkv=nkv, dk=dk, dv=dv, page_size=P_, nsplit=2, split_stride=proj.stride(0), status=status,
                         per_head=True, q_temp=temp, v_scale=0.6)
    tol = 5e-6 if dtype == torch.float32 else 1e-2
    t = P.query_temperature(positions, None if temp is None else dict(coef=temp[0], every=temp[1]))
    close(q.view(T, nq, dk), P.unit(p[:, :nq * dk].reshape(T, nq, dk), 1e-4) * t[:, None, None], tol, "q")
    k = P.unit(p[:, nq * dk:(nq + nkv) * dk].reshape(T, nkv, dk), 1e-4)
    v = 0.6 * p[:, (nq + nkv) * dk:wide].reshape(T, nkv, dv)
    for i, pos in enumerate(positions):
        page = cache[int(pages[pos // P_])]
        kp, vp = page[:nkv * P_ * dk].view(nkv, P_, dk), page[nkv * P_ * dk:].view(nkv, P_, dv)
        close(kp[:, pos % P_], k[i], tol, "k")
        close(vp[:, pos % P_], v[i], tol, "v")
    assert int(status) == 0


@pytest.mark.parametrize("M,N,Kd", [(200, 4096, 256), (1500, 1000, 136), (130, 16384, 64), (1100, 2064, 520)])
def test_gelu_in_the_products_epilogue(M, N, Kd):
    from mini_hisparse_b200.kernels.runtime import make_runtime
    from mini_hisparse_b200.parts import Workspace

    rt = make_runtime("cuda:0", torch.bfloat16)
    rt.status = torch.zeros(1, dtype=torch.int32, device="cuda")
    g = torch.Generator().manual_seed(M)
    x, w = torch.randn(M, Kd, generator=g).bfloat16(), (torch.randn(N, Kd, generator=g) * 2 / Kd ** 0.5).bfloat16()
    out = rt.linear_act(x.cuda(), w.cuda(), "gelu_tanh", Workspace(rt.device), "a")
    ref = P.gelu_tanh(x.double() @ w.double().T)
    assert out.dtype == torch.bfloat16 and int(rt.status) == 0
    torch.testing.assert_close(out.double().cpu(), ref, atol=1e-3, rtol=5e-3)


# ---- the mixers alone, over inputs made by hand --------------------------------------------------------------
class MixerRun:
    """One mixer over a cache of its own; feed() brings some requests' next input rows and returns theirs."""

    def __init__(self, spec, tensors, dtype, page_size=16, pages=40):
        from mini_hisparse_b200.parts import MIXERS
        from test_parts_gpu import harness

        needs = MIXERS.build(spec)
        sides = needs.side_needs()
        self.rt, self.cache, self.batch, self.ws, self.status = harness([needs.cache_need(), *sides.values()], dtype, pages, page_size)
        self.mixer = MIXERS.build(spec, rt=self.rt)
        self.mixer.load({k: t.to("cuda", torch.float32 if self.mixer.parameters()[k].role == "vector" else dtype)
                         for k, t in tensors.items()})
        self.user = self.batch.add_user(0, self.mixer)
        self.sides = {n: self.batch.add_user(1 + i, self.mixer.side_user(n)) for i, n in enumerate(sides)}
        self.dtype = dtype

    def feed(self, rows):
        from mini_hisparse_b200.engine import StepEntry
        from test_parts_gpu import context

        for r in rows:
            if r not in self.cache.requests:
                self.cache.open(r)
        ctx, views, _ = context(self.rt, self.cache, self.batch, self.ws, self.status, [StepEntry(r, [0] * len(h), []) for r, h in rows.items()])
        view = self.batch.cache_view(self.user, views)
        view.sides = {n: self.batch.cache_view(u, views) for n, u in self.sides.items()}
        out = self.mixer.forward(torch.cat(list(rows.values())).to("cuda", self.dtype), ctx, view).reduced().cpu()
        got, at = {}, 0
        for r, h in rows.items():
            got[r] = out[at:at + len(h)]
            at += len(h)
            self.cache.advance(r, len(h))
        assert int(self.status) == 0
        return got

    def sequence(self, h, cuts):
        """One request alone, in portions of the given sizes."""
        out, at = [], 0
        for n in cuts:
            out.append(self.feed({"a": h[at:at + n]})["a"])
            at += n
        assert at == len(h)
        self.cache.close("a")
        return torch.cat(out)


CUTS = {"whole": lambda n: [n], "decode": lambda n: [n - 20] + [1] * 20, "portions": lambda n: [n - 81, 2, 17, 3, 40, 16, 2, 1],
        "alone": lambda n: [1] * n}


@pytest.mark.parametrize("H,G,d,dv,P_,dtype", [(6, 3, 24, 40, 16, torch.float32), (4, 2, 64, 64, 16, torch.bfloat16),
                                               (8, 1, 128, 128, 32, torch.bfloat16), (6, 3, 24, 40, 16, torch.bfloat16),
                                               (2, 2, 20, 20, 8, torch.bfloat16), (4, 2, 64, 64, 24, torch.bfloat16)])
def test_attention_finds_one_key_among_hundreds(H, G, d, dv, P_, dtype):
    """Projections that pick columns of the input, so that q, k and v are what the test says.  In 300 positions of which
    the last 60 queries each look for ONE key (its score stands out by far): the first position, the last of a page and
    the first of the next, a key far back, the one before the query and the query's own; every cut; and a request beside
    another."""
    from mini_hisparse_b200.parts import PartSpec

    L, wide = 300, H * d + G * (d + dv) + H
    g = torch.Generator().manual_seed(d)
    h = torch.randn(L, wide, generator=g).bfloat16().float()
    targets = [0, 1, P_ - 1, P_, 2 * P_ - 1, 63, 64, 127, 128, 200]
    q0, k0 = 0, H * d
    for i in range(240, L):
        j = (targets + [i - 1, i])[(i - 240) % 12]
        for hd in range(H):
            key = h[j, k0 + hd // (H // G) * d:][:d]
            h[i, q0 + hd * d:q0 + (hd + 1) * d] = key
    eye = torch.eye(wide)
    out = torch.randn(48, H * dv, generator=g) / (H * dv) ** 0.5
    tensors = {"q": eye[:H * d], "k": eye[k0:k0 + G * d], "v": eye[k0 + G * d:k0 + G * (d + dv)], "g": eye[wide - H:], "o": out}
    m = dict(heads=H, kv_heads=G, dim=d, vdim=dv, scale=16.0 / d, q_temp=dict(coef=0.3, every=100))
    w = {k: t.to(dtype).double() for k, t in tensors.items()}
    ref = 0.75 * P.attention(h.double(), w, "", m, 1e-5)
    spec = PartSpec.make("unit_attention", hidden_size=wide, q_heads=H, kv_heads=G, dim=d, vdim=dv, scale=m["scale"], eps=1e-5,
                         q_temp=(0.3, 100), out_scale=0.75, position=PartSpec.make("none"))
    run = MixerRun(spec, tensors, dtype, page_size=P_, pages=2 * -(-L // P_) + 1)
    tol = 2e-5 if dtype == torch.float32 else 0.03
    for name, cut in CUTS.items():
        close(run.sequence(h, cut(L)), ref, tol, name)
    both = run.feed({"a": h[:250], "b": h[:1]})
    more = run.feed({"b": h[1:120], "a": h[250:251]})
    last = run.feed({"a": h[251:L], "b": h[120:121]})
    close(torch.cat((both["a"], more["a"], last["a"])), ref, tol, "beside another")
    close(torch.cat((both["b"], more["b"], last["b"])), ref[:121], tol, "the other")


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_the_scan_remembers_one_token(dtype):
    """Slow decays and one input a hundred times larger than the rest, in the first token: its write is what the outputs
    hold 400 tokens later, whatever the cuts; a neighbour request without it differs by far."""
    from mini_hisparse_b200.parts import PartSpec

    hidden, inner, N, R, taps, L = 64, 56, 9, 4, 4, 420
    g = torch.Generator().manual_seed(4)
    t = {"in": torch.randn(2 * inner, hidden, generator=g) / 8, "conv": torch.randn(inner, taps, generator=g) * 0.5,
         "conv.b": torch.randn(inner, generator=g) * 0.1, "x": torch.randn(R + 2 * N, inner, generator=g) / 7,
         "dt": torch.randn(inner, R, generator=g) * 0.1, "dt.b": torch.full((inner,), -4.0),
         "A_log": torch.full((inner, N), -3.0), "D": torch.randn(inner, generator=g), "o": torch.randn(48, inner, generator=g) / 7}
    t = {k: v.bfloat16().float() for k, v in t.items()}
    h = torch.randn(L, hidden, generator=g).bfloat16().float()
    big = h.clone()
    big[0] *= 30
    m = dict(inner=inner, state=N, dt_rank=R, conv=taps)
    w = {k: v.double() for k, v in t.items()}
    refs = {"a": P.selective_scan(big.double(), w, "", m, 0), "b": P.selective_scan(h.double(), w, "", m, 0)}
    apart = float((refs["a"][-1] - refs["b"][-1]).abs().max()) / float(refs["b"].abs().max())
    assert apart > 0.05
    spec = PartSpec.make("selective_scan", hidden_size=hidden, inner=inner, state=N, dt_rank=R, conv=taps)
    run = MixerRun(spec, t, dtype)
    for name, cut in CUTS.items():
        got = run.sequence(big, cut(L))
        close(got[-100:], refs["a"][-100:], 2e-5 if dtype == torch.float32 else 0.02, name)
    one, two = run.feed({"a": big[:300], "b": h[:2]}), run.feed({"b": h[2:3], "a": big[300:]})
    close(torch.cat((one["a"], two["a"]))[-100:], refs["a"][-100:], 2e-5 if dtype == torch.float32 else 0.02, "beside another")
    close(torch.cat((one["b"], two["b"])), refs["b"][:3], 2e-5 if dtype == torch.float32 else 0.02, "the other")


# ---- the model through the step function ---------------------------------------------------------------------
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_schedule_agrees_with_the_plain_model(models, name, dtype):
    """Whole prompts; most of a prompt and then its tail token by token, three requests side by side (captured graphs);
    portions of changing size down to two tokens; mixed batches with up to four live requests over a pool that holds no
    more than they need, so that pages and slots are used again (freed pages are poisoned).  Every position is compared."""
    folder, cfg, w = models[name]
    reqs = requests_for(cfg, [150, 1, 23, 97, 64, 2, 131])
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    whole = None
    for steps in (S.whole(reqs), S.tail_one_by_one(reqs, tail=45), S.changing_portions(reqs), S.mixed(reqs, seed=3)):
        got, runner, cache = run_steps(folder, dtype, steps, page_size=PAGES[name])
        check_against_plain(got, refs, dtype)
        whole = whole or got
        check_rows(torch.cat([row_errors(got[rid], whole[rid]) for rid in reqs]), dtype)
    assert all(g["pages_reused"] > 0 for g in cache["page_groups"])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_the_stream_after_every_layer(models, dtype):
    """The residual stream after every layer run (a repeated layer counts each time), what is pending added."""
    from mini_hisparse_b200 import CacheConfig, CacheManager, load_model
    from mini_hisparse_b200.engine import ModelRunner, StepEntry

    folder, cfg, w = models["A"]
    toks = random_tokens(cfg["vocab"], 75, 12)
    _, streams = P.forward(cfg, w, toks, return_layers=True)
    model_ = load_model(folder, dtype=dtype)
    cache = CacheManager(model_.cache_needs, CacheConfig(num_pages=8, page_size=16, max_requests=2, dtype=model_.rt.dtype))
    runner = ModelRunner(model_, cache, use_graphs=False)
    seen = {}

    def observer(i, x, pending):
        seen[i] = (x + pending.reduced() if pending is not None else x).float().cpu().clone()

    runner.observer = observer
    cache.open("a")
    runner.step([StepEntry("a", toks, [len(toks) - 1])])
    assert [i for i in seen if i != "final"] == list(range(len(P.run_order(cfg)))) == list(range(8))
    for i in range(8):
        err = float(row_errors(seen[i], streams[i]).max())
        assert err < (1e-5 if dtype == "float32" else 0.04), f"after layer run {i}: {err:.3g}"
    torch.testing.assert_close(seen["final"], seen[7], atol=1e-5, rtol=1e-5)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_tokens_reach_the_last_logits(tmp_path, dtype):
    """Requests of 700 tokens; a changed third token moves the plain model's last logits by more than the float32 tolerance,
    so a lost page or state shows.  Decoded tokens and short portions far into it, every cut against the plain model."""
    from mini_hisparse_b200 import write_random_model

    cfg = model(120, 128, [parallel(left(4, 2, 32, 32, scale=0.4, temp=(0.3, 64)), right(96, 16, 8, 4), ff=128), gru(96, ff=128),
                           parallel(left(4, 2, 64, 64, scale=0.2), right(64, 8, 8, 4), ff=96)], loop=(0, 2, 2))
    write_random_model(cfg, 31, tmp_path, dtype=torch.bfloat16, matrix_std=0.1)
    cfg, w = P.load_folder(tmp_path)
    reqs = requests_for(cfg, [700], seed=70)
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    changed = list(reqs["r0"])
    changed[2] = (changed[2] + 1) % cfg["vocab"]
    assert float(row_errors(P.forward(cfg, w, changed)[-1:].float(), refs["r0"][-1:])) > 5 * F32_ROW
    for steps in (S.whole(reqs), S.tail_one_by_one(reqs, tail=40), S.changing_portions(reqs, sizes=(530, 2, 7, 64, 3, 2))):
        got, stats, pages = run_steps(tmp_path, dtype, steps)
        check_against_plain(got, refs, dtype)


def test_the_plain_model_is_sensitive_to_what_the_tests_are_for(models):
    """A temperature that steps one position off, factors, filters turned around, a state that starts elsewhere, a pass
    without its vector or without the embedding output: each moves the plain model's logits by far more than the float32
    tolerance, so the comparisons above would show them."""
    folder, cfg, w = models["A"]
    toks = random_tokens(cfg["vocab"], 90, 5)
    right_ = P.forward(cfg, w, toks)
    rms = float(right_.pow(2).mean().sqrt())

    def moved(cfg2=None, w2=None):
        return float((P.forward(cfg2 or cfg, w2 or w, toks) - right_).pow(2).mean().sqrt()) / rms

    changes = [lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(every=8),
               lambda c: c["layers"][0]["mixer"]["left"]["q_temp"].update(coef=0.3),
               lambda c: c["layers"][3]["mixer"]["left"].update(q_temp=dict(coef=0.1, every=30)),
               lambda c: c["layers"][0]["mixer"].update(left_scale=0.6), lambda c: c["layers"][3]["mixer"].update(right_scale=0.5),
               lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.35), lambda c: c["loop"].update(times=1),
               lambda c: c["embedding"].update(scale=2.9)]
    for change in changes:
        c = copy.deepcopy(cfg)
        change(c)
        assert moved(c) > 20 * F32_ROW
    for name, fn in (("l0.canon1", lambda t: t.flip(-1)), ("l1.canon2", lambda t: t * 0), ("l0.mix.right.conv", lambda t: t.flip(-1)),
                     ("l0.mix.right.A_log", lambda t: t + 0.5), ("l0.mix.right.D", lambda t: t * 0),
                     ("l0.mix.right.dt.b", lambda t: t + 0.3), ("l1.mix.z.b", lambda t: t * 0), ("l1.mix.x.b", lambda t: t * 0),
                     ("loop.step", lambda t: t.flip(0)), ("l0.norm1.alpha", lambda t: t * 1.2), ("final.norm.b", lambda t: t * 0)):
        w2 = dict(w)
        w2[name] = fn(w[name])
        assert moved(w2=w2) > 20 * F32_ROW, name


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_a_slot_used_again(models, dtype):
    """A short prompt, then 260 tokens one by one, two requests side by side; then their slots and pages serve new
    requests, whose states and kept inputs must start from zero."""
    folder, cfg, w = models["A"]
    reqs = requests_for(cfg, [270, 265], seed=40)
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    steps = S.tail_one_by_one(reqs, tail=260, together=2)
    again = {f"again_{k}": v for k, v in requests_for(cfg, [50, 31], seed=60).items()}
    refs.update({rid: P.forward(cfg, w, toks).float() for rid, toks in again.items()})
    steps += S.changing_portions(again, sizes=(2, 29, 1, 7))
    got, runner, cache = run_steps(folder, dtype, steps, max_requests=2)
    check_against_plain(got, refs, dtype)
    assert runner["graph_steps"] > 200


def test_batches_of_unequal_requests_equal_each_alone(models):
    """float32: a request's logits in a mixed batch equal those it gets alone, to rounding."""
    folder, cfg, w = models["C"]
    reqs = requests_for(cfg, [140, 3, 77, 30], seed=9)
    alone, _, _ = run_steps(folder, "float32", S.whole(reqs), page_size=16)
    mixed, _, _ = run_steps(folder, "float32", S.mixed(reqs, seed=11, tail=20), page_size=16)
    for rid in reqs:
        assert row_rms_error(mixed[rid], alone[rid]) < F32_ROW


def test_a_model_without_pages(tmp_path):
    """Only minGRU layers: nothing is kept in pages, and every schedule works on state slots alone."""
    from mini_hisparse_b200 import write_random_model

    cfg = model(80, 72, [gru(48, ff=64), gru(80)], taps=2, loop=(1, 2, 2))
    write_random_model(cfg, 3, tmp_path, dtype=torch.bfloat16, matrix_std=0.15)
    cfg, w = P.load_folder(tmp_path)
    reqs = requests_for(cfg, [60, 33, 1, 20, 41], seed=2)
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    for steps in (S.tail_one_by_one(reqs, tail=12), S.mixed(reqs, seed=5)):
        got, _, cache = run_steps(tmp_path, "float32", steps)
        check_against_plain(got, refs, "float32")
    assert cache["page_groups"] == []


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_an_input_convolution_behind_another_norm(dtype):
    """The arrangement with an RMS norm: norm and convolution are two kernels and the stream stays where it is."""
    from mini_hisparse_b200.engine import StepEntry
    from mini_hisparse_b200.parts import LayerSpec, PartSpec
    from mini_hisparse_b200.parts.registry import BLOCKS
    from test_parts_gpu import context, harness

    dt = torch.float32 if dtype == "float32" else torch.bfloat16
    W = 64
    norm, conv = PartSpec.make("rmsnorm", width=W, eps=1e-5), PartSpec.make("causal_conv", width=W, taps=3)
    spec = LayerSpec.make("l", "pre_norm_conv", {"mixer_norm": norm, "mixer_conv": conv,
                                                 "mixer": PartSpec.make("mingru", hidden_size=W, width=40)})
    block = BLOCKS.get(spec.block)(spec, None)
    rt, cache, batch, ws, status = harness([block.cache_need(), *block.side_needs().values()], dt)
    block = BLOCKS.get(spec.block)(spec, rt)
    g = torch.Generator().manual_seed(8)
    w = {}
    for role, part in block.parts().items():
        t = {k: (torch.randn(ps.shape, generator=g) * 0.3).bfloat16().float() for k, ps in part.parameters().items()}
        w[role] = {k: v.double() for k, v in t.items()}
        part.load({k: v.to("cuda", torch.float32 if part.parameters()[k].role == "vector" else dt) for k, v in t.items()})
    users = [batch.add_user(0, block), batch.add_user(1, None)]
    x = torch.randn(50, W, generator=g)
    n = P.unit(x.double(), 1e-5) * w["mixer_norm"]["weight"]
    ref = P.mingru(P.with_convolution(n, w["mixer_conv"]["weight"]), w["mixer"], "", None, None)
    cache.open("a")
    at = 0
    for count in (20, 1, 2, 27):
        ctx, views, _ = context(rt, cache, batch, ws, status, [StepEntry("a", [0] * count, [])])
        view = batch.cache_view(users[0], views)
        view.sides = {"input_conv": batch.cache_view(users[1], views)}
        xd = x[at:at + count].cuda()
        out = block.forward(xd, None, ctx, view).reduced()
        assert ctx.extras["stream"].data_ptr() == xd.data_ptr()
        close(out, ref[at:at + count], 2e-5 if dtype == "float32" else 0.03, f"rows {at} ...")
        cache.advance("a", count)
        at += count


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(models, dtype):
    """Engine.add_request / run: admission, portions under a token budget, decoding, finishing.  float32 tokens equal the
    plain model's; in bfloat16 every token is the plain model's choice for the engine's own history, or loses to it by
    less than rounding."""
    from mini_hisparse_b200 import Engine, load_model

    folder, cfg, w = models["A"]
    model_ = load_model(folder, dtype=dtype)
    engine = Engine(model_, num_pages=40, page_size=16, max_requests=3, max_tokens_per_step=48, graph_after=2)
    prompts = requests_for(cfg, [70, 9, 33, 12], seed=80)
    for rid, p in prompts.items():
        engine.add_request(rid, p, max_new_tokens=12)
    out = engine.run()
    engine.cache.assert_invariants()
    for rid, p in prompts.items():
        assert len(out[rid]) == 12
        if dtype == "float32":
            assert out[rid] == P.generate(cfg, w, p, 12)
        else:
            seq = list(p)
            for tok in out[rid]:
                logits = P.forward(cfg, w, seq)[-1]
                assert float(logits.max() - logits[tok]) < 0.08 * float(logits.abs().max())
                seq.append(tok)


def test_command_line_demo_with_a_zetenex_config(capsys):
    """`demo --config configs/zetenex-demo.json`: random weights, three requests through Engine and scheduler."""
    from pathlib import Path

    import mini_hisparse_b200
    from mini_hisparse_b200 import cli

    config = Path(mini_hisparse_b200.__file__).parent / "configs" / "zetenex-demo.json"
    assert cli.main(["demo", "--config", str(config), "--dtype", "bfloat16", "--requests", "3", "--prompt-tokens", "70",
                     "--max-new-tokens", "6"]) == 0
    report = json.loads(capsys.readouterr().out)
    assert [r["generated_tokens"] for r in report["requests"].values()] == [6, 6, 6]


def test_trace_run_picks_the_model_by_its_config(models, tmp_path):
    """bin/trace_run on a Zetenex folder: the same program, cache and step function as for every model."""
    folder, cfg, w = models["D"]
    reqs = requests_for(cfg, [60, 21], seed=90)
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    steps = S.mixed(reqs, seed=1, tail=10)
    run = TraceRun(folder, "float32", tmp_path / "out", S.peak_tokens(steps), page_size=16, extra=("--poison",))
    got = {}
    for entries, end in steps:
        logits = run.step(entries, end)
        row = 0
        for e in entries:
            got.setdefault(e["id"], []).append(logits[row: row + len(e["want"])])
            row += len(e["want"])
    assert run.close() == 0
    check_against_plain({k: torch.cat(v) for k, v in got.items()}, refs, "float32")
