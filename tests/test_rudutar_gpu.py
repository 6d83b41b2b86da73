"""Rudutar through the engine against the plain implementation of tests/plain/rudutar_plain.py.

Small configurations made here (none is anyone's model), random weights from a seed.  Covered: the kernels of each
mechanism alone (the normalised gather; convolution, norms, temperature and append over segments that start, go on and
end anywhere, in both kernels; keys that are values too, with biases; distance biases, the constant sink and the window
in every attention kernel, with one key made to stand out just inside and just outside the window, at page borders and at
the start of a sequence; the router's scores, groups and weights; relu-squared experts with an ungated shared one; the
activations in the product's epilogue); whole prompts; prefill against token-by-token decoding through captured graphs;
portions down to two tokens; mixed batches over a tight pool whose freed pages are poisoned; slots used again; long
decoding; sizes that are equal or 1; readers with wider and narrower windows than the layer they read; generation through
Engine and its scheduler; the command line; bin/trace_run.
"""
import copy
import json

import pytest
import torch

import schedules as S
from conftest import TraceRun, random_tokens, row_rms_error
from plain import rudutar_plain as P
from test_dotivik_gpu import Parts, dev_i, run_steps

pytestmark = pytest.mark.gpu


def sloped(heads, kv_heads, dim, vdim, conv, size, temp=(0.4, 9), scale=0.3, kv_from=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv, scale=scale, mask=dict(size=size))
    if temp is not None:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def keyed(heads, kv_heads, dim, size, rot=None, base=3000.0, scale=0.3):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=scale, mask=dict(size=size))
    if rot is not None:
        m["rot"] = dict(dims=rot, base=base)
    return m


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, scale=1.3, groups=None, shared=None):
    out = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if groups is not None:
        out["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared is not None:
        out["shared"] = dict(ff=shared)
    return out


def layer(kind, mixer, mlp=None):
    return dict(type=kind, mixer=mixer, mlp=mlp)


def model(vocab, width, layers, eps=1e-5):
    return dict(architecture="Rudutar", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)


# A: every branch at once, with windows that prompts of a hundred tokens pass many times: values wider than keys, a reader
# with a wider window than the layer it reads and one with a narrower, a layer without a feed-forward, groups of two and
# of four experts, a shared expert and none, a temperature with a step that is no integer.
CFG_A = model(203, 96, [
    layer("attention", sloped(6, 3, 24, 40, 4, 21), dense(160)),
    layer("attention_2", keyed(4, 2, 40, 13, rot=16), moe(8, 2, 32, groups=(4, 2), shared=56)),
    layer("attention", sloped(3, 3, 24, 40, 2, 34, temp=None, kv_from=0), moe(8, 3, 24, groups=(2, 1))),
    layer("attention", sloped(6, 3, 24, 40, 3, 8, temp=(0.7, 5.5), kv_from=0), None),
    layer("attention_2", keyed(6, 6, 16, 27, rot=16, base=50.0), dense(72)),
    layer("attention", sloped(4, 1, 32, 16, 3, 30), moe(5, 2, 40, scale=0.6, shared=24))])
# B: values that a usual model makes different are equal or 1 here: one head, as many KV heads as heads, windows of one
# and two positions, filters of one tap and of seven, no rotation, a single expert, groups of one expert, all groups kept,
# a temperature step of 1, a width that no tensor-core product takes.
CFG_B = model(97, 100, [
    layer("attention", sloped(1, 1, 20, 20, 1, 1, temp=(0.3, 1)), moe(1, 1, 20, scale=1.0)),
    layer("attention_2", keyed(1, 1, 12, 2), dense(12)),
    layer("attention", sloped(3, 3, 12, 8, 7, 10), moe(4, 2, 16, groups=(4, 2), shared=4)),
    layer("attention_2", keyed(5, 1, 20, 9, rot=20, base=100.0), moe(6, 6, 8, groups=(3, 3))),
    layer("attention", sloped(3, 3, 12, 8, 5, 10, kv_from=2), dense(28))], eps=1e-3)
# C: sizes of a real model's order: heads of 128 and of 64 (the tcgen05 and TMA kernels), windows of some hundred.
CFG_C = model(300, 256, [
    layer("attention", sloped(8, 2, 64, 64, 4, 96, temp=(0.2, 64), scale=0.12), dense(512)),
    layer("attention_2", keyed(4, 2, 128, 80, rot=64, base=1e6, scale=0.09), moe(16, 4, 128, groups=(4, 2), shared=128)),
    layer("attention", sloped(4, 2, 64, 64, 4, 70, kv_from=0, scale=0.12), moe(16, 2, 64, groups=(8, 3), shared=64)),
    layer("attention", sloped(4, 1, 128, 128, 2, 64, scale=0.09), dense(384))])
CONFIGS = {"A": CFG_A, "B": CFG_B, "C": CFG_C}
PAGES = {"A": 16, "B": 8, "C": 32}
# A row's error: the root mean square of (got - plain) as a share of the row's root mean square.  float32: computed in
# float64 by the plain model; any order of float32 sums differs from that by about 1e-6.  bfloat16: the median row is held
# tightly (a fault in a kernel moves all rows); single rows may take another expert than the plain model, because the
# router reads the bfloat16 rounding of its input, so the share of rows that are far off is bounded, and every schedule is
# compared with the whole prompt in the same dtype in the same way.
BF16_MEDIAN, BF16_FAR, BF16_FAR_SHARE = 0.02, 0.15, 0.1
F32_MEAN, F32_ROW = 5e-6, 1e-4


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    from mini_hisparse_b200 import write_random_model

    out = {}
    for name, cfg in CONFIGS.items():
        folder = tmp_path_factory.mktemp(f"rudutar{name}")
        write_random_model(cfg, 43, folder, dtype=torch.bfloat16, matrix_std=0.15)
        out[name] = (folder, *P.load_folder(folder))
    return out


def requests_for(cfg, lengths, seed=0):
    return {f"r{i}": random_tokens(cfg["vocab"], n, seed + i) for i, n in enumerate(lengths)}


def row_errors(got, ref):
    return (got.double() - ref.double()).pow(2).mean(-1).sqrt() / ref.double().pow(2).mean(-1).sqrt()


def check_rows(err, dtype):
    if dtype == "float32":
        assert float(err.mean()) < F32_MEAN and float(err.max()) < F32_ROW, \
            f"mean row error {float(err.mean()):.3g}, worst {float(err.max()):.3g} at {int(err.argmax())} of all rows"
    else:
        far = float((err > BF16_FAR).double().mean())
        assert float(err.median()) < BF16_MEDIAN and far < BF16_FAR_SHARE, \
            f"median row error {float(err.median()):.3g}, {far:.3g} of the rows beyond {BF16_FAR}"


def check_against_plain(got, refs, dtype):
    for rid, ref in refs.items():
        assert got[rid].shape == ref.shape
    check_rows(torch.cat([row_errors(got[rid], ref) for rid, ref in refs.items()]), dtype)


def close(got, ref, tol, what=""):
    ref = ref.double()
    err = float((got.double().cpu() - ref).abs().max())
    assert err < tol * float(ref.abs().max()), f"{what}: {err:.3g} beside values up to {float(ref.abs().max()):.3g}"


class Batch:
    """A step's segments as the kernels' wrappers read them: counts, first positions and slots."""

    def __init__(self, counts, starts, slots):
        self.counts, self.starts, self.slots = counts, starts, slots
        self.T = sum(counts)
        self.offsets = [sum(counts[:i]) for i in range(len(counts) + 1)]
        self.seg_offset, self.seg_slot = dev_i(self.offsets), dev_i(slots)
        self.positions = dev_i([s + i for s, n in zip(starts, counts) for i in range(n)])
        self.segments, self.longest = counts, max(counts)
        self.status = torch.zeros(1, dtype=torch.int32, device="cuda")

    def rows(self, i):
        return slice(self.offsets[i], self.offsets[i + 1])


# segments that start a sequence, go on after few or many tokens, hold one token, fewer than a filter's taps, exactly a
# tile of the kernel, one more, and several tiles; slots in no order
BATCHES = [([1, 2, 5, 16, 17, 40, 3], [0, 9, 0, 4, 0, 1, 2], [5, 0, 3, 6, 1, 2, 4]), ([1, 1, 1], [0, 7, 1], [2, 0, 1]),
           ([70], [0], [0]), ([33], [50], [1])]


# ---- the kernels of each mechanism alone --------------------------------------------------------------------
@pytest.mark.parametrize("H", [100, 2048])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gather_with_a_norm(H, dtype):
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(H)
    table, w = torch.randn(11, H, generator=g).to(dtype), 1 + 0.1 * torch.randn(H, generator=g)
    out, status = torch.empty(5, H, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
    K.embed_norm(table.cuda(), w.cuda(), 0.1, dev_i([3, 10, 0, 3, 7]), out, status=status)
    close(out, P.unit_rms(table[[3, 10, 0, 3, 7]].double(), 0.1) * w.double(), 2e-6)
    assert int(status) == 0
    K.embed_norm(table.cuda(), w.cuda(), 0.1, dev_i([3, 11, 0, -1, 7]), out, status=status)      # reported, zeros
    assert int(status) == 1 and float(out[[1, 3]].abs().max()) == 0


@pytest.mark.parametrize("nq,nkv,dk,dv,taps,has_kv,P_", [
    (6, 3, 24, 40, 4, True, 16), (3, 3, 24, 40, 2, False, 16), (1, 1, 20, 20, 1, True, 8), (2, 1, 128, 64, 3, True, 32),
    (3, 3, 12, 8, 7, True, 7), (2, 2, 18, 33, 3, True, 16), (4, 1, 136, 200, 4, True, 16), (5, 1, 32, 32, 16, False, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("batch", range(len(BATCHES)))
def test_convolved_heads(nq, nkv, dk, dv, taps, has_kv, P_, dtype, batch):
    """Convolution over a step's edge with the slot's kept rows (a fresh sequence sees none, whatever its slot holds), the
    norm of each head, the temperature at and beside its steps, q's rows and the pages of k and v, the renewed kept rows;
    slots and pages of others stay as they are."""
    from mini_hisparse_b200.kernels import api as K

    b = Batch(*BATCHES[batch])
    g = torch.Generator().manual_seed(nq * dk + taps)
    eps, temp, nsplit = 1e-5, (0.5, 4), 2
    qw, kw, vw = nq * dk, nkv * dk, nkv * dv
    C = qw + (kw + vw if has_kv else 0)
    ld = -(-(C + 5) // 16) * 16
    proj = torch.randn(nsplit, b.T, ld, generator=g)
    z = proj.double().sum(0)
    filt = torch.randn(C, taps, generator=g) * 0.6
    wq, wk = 1 + 0.2 * torch.randn(dk, generator=g), 1 + 0.2 * torch.randn(dk, generator=g)
    keep0 = torch.randn(7, max(taps - 1, 1), C, generator=g)
    ref_keep = keep0.double().clone()
    longest = max(s + n for s, n in zip(b.starts, b.counts))
    n_pages = -(-longest // P_)
    table = torch.randperm(len(b.counts) * n_pages + 2, generator=g)[:len(b.counts) * n_pages].view(len(b.counts), n_pages)
    page_elems = nkv * P_ * (dk + dv)
    pool = torch.full((table.numel() + 2, page_elems), 7.0, dtype=dtype, device="cuda")
    before = pool.clone()
    keep, q_out, pd = keep0.cuda(), torch.empty(b.T, qw, dtype=dtype, device="cuda"), proj.cuda()
    K.head_conv_append(Parts(pd, nsplit), filt.t().contiguous().cuda(), wq.cuda(), wk.cuda() if has_kv else None, eps,
                       keep if taps > 1 else None, b, dev_i(table), q_out, pool, nq=nq, nkv=nkv, dk=dk, dv=dv, page_size=P_,
                       has_kv=has_kv, q_temp=temp)
    assert int(b.status) == 0
    tol = 3e-6 if dtype == torch.float32 else 0.006
    st, touched = pool.float().cpu().double(), torch.zeros(pool.shape, dtype=torch.bool)
    for i, (n, start, slot) in enumerate(zip(b.counts, b.starts, b.slots)):
        rows = z[b.rows(i), :C]
        held = keep0[slot].double()[:taps - 1] if start else torch.zeros(taps - 1, C, dtype=torch.float64)
        both = torch.cat((held, rows), 0)
        y = P.short_convolution(both, filt.double())[taps - 1:]
        pos = torch.arange(start, start + n)
        q = P.unit_rms(y[:, :qw].view(n, nq, dk), eps) * wq.double() * P.temperature(pos, *temp)[:, None, None]
        close(q_out[b.rows(i)].float().view(n, nq, dk), q, tol, f"q of segment {i}")
        if taps > 1:
            ref_keep[slot, :taps - 1] = both[n:]
        if not has_kv:
            continue
        k = P.unit_rms(y[:, qw:qw + kw].view(n, nkv, dk), eps) * wk.double()
        v = y[:, qw + kw:].view(n, nkv, dv)
        for t in range(n):
            page, w = int(table[i, (start + t) // P_]), (start + t) % P_
            kp, vp = st[page, :nkv * P_ * dk].view(nkv, P_, dk)[:, w], st[page, nkv * P_ * dk:].view(nkv, P_, dv)[:, w]
            touched[page, :nkv * P_ * dk].view(nkv, P_, dk)[:, w] = True
            touched[page, nkv * P_ * dk:].view(nkv, P_, dv)[:, w] = True
            close(kp, k[t], tol * 2, "a cached key")
            close(vp, v[t], tol * 2, "a cached value")
    if taps > 1:
        close(keep, ref_keep, 1e-6, "kept rows")
        others = [s for s in range(7) if s not in b.slots]
        assert torch.equal(keep[others].cpu(), keep0[others])
    assert torch.equal(pool.cpu()[~touched], before.cpu()[~touched])


@pytest.mark.parametrize("nq,nkv,dk,rdim,P_,ld_extra", [(4, 2, 40, 16, 16, 4), (1, 1, 12, 0, 8, 1), (5, 1, 20, 20, 7, 5), (4, 2, 128, 64, 32, 4)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_keys_that_are_values(nq, nkv, dk, rdim, P_, ld_extra, dtype):
    """Biases join q and k before everything else; the values are k as projected (bias included, neither normalised nor
    rotated), beside the normalised and rotated keys."""
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(nq * dk)
    T, nsplit, eps, start = 21, 2, 1e-5, 30
    qw, kw = nq * dk, nkv * dk
    proj, bias = torch.randn(nsplit, T, qw + kw + ld_extra, generator=g), torch.randn(qw + kw, generator=g)
    wq, wk = 1 + 0.2 * torch.randn(qw, generator=g), 1 + 0.2 * torch.randn(kw, generator=g)
    z = proj.double().sum(0)[:, :qw + kw] + bias.double()
    pos = torch.arange(start, start + T)
    q = (P.unit_rms(z[:, :qw], eps) * wq.double()).view(T, nq, dk)
    k = (P.unit_rms(z[:, qw:], eps) * wk.double()).view(T, nkv, dk)
    inv = None
    if rdim:
        q, k = P.rotate_half_split(q, pos, rdim, 700.0), P.rotate_half_split(k, pos, rdim, 700.0)
        inv = (700.0 ** (-torch.arange(0, rdim, 2, dtype=torch.float64) / rdim)).float().cuda()
    table = torch.randperm(12, generator=g)[None]
    pool = torch.zeros(12, nkv * P_ * 2 * dk, dtype=dtype, device="cuda")
    q_out, pd = torch.empty(T, qw, dtype=dtype, device="cuda"), proj.cuda()
    K.qknorm_rope_append(pd, wq.cuda(), wk.cuda(), eps, dev_i(pos), dev_i([0] * T), dev_i(table), inv, rdim, q_out, pool, nq=nq,
                         nkv=nkv, dk=dk, dv=dk, page_size=P_, nsplit=nsplit, split_stride=pd.stride(0), bias=bias.cuda(),
                         v_from_k=True)
    tol = 3e-6 if dtype == torch.float32 else 0.005
    close(q_out.float().view(T, nq, dk), q, tol, "q")
    st = pool.float().cpu().double()
    for t in range(T):
        page, w = int(table[0, (start + t) // P_]), (start + t) % P_
        close(st[page, :nkv * P_ * dk].view(nkv, P_, dk)[:, w], k[t], tol * 2, "key")
        close(st[page, nkv * P_ * dk:].view(nkv, P_, dk)[:, w], z[t, qw:].view(nkv, dk), tol * 2, "value")


def attend(kernel, pool, table, q, segs, *, H, G, d, dv, P_, window, scale, sms, dtype, gate=None, per_head=False, **opts):
    """The plan's items of one request's segments on one of the kernels and, where it applies, the merge of key splits."""
    from mini_hisparse_b200.kernels import api as K
    from mini_hisparse_b200.parts.attention import AttentionShape, plan_attention

    T = sum(s.count for s in segs)
    plan = plan_attention(AttentionShape(H, G, window, {"tc": 128, "mma": 64, "simt": 16}[kernel]), segs, T, sm_count=sms)
    part_acc = torch.empty(max(1, plan.part_rows), H, dv, device="cuda")
    part_ml = torch.empty(max(1, plan.part_rows), H, 2, device="cuda")
    o = torch.zeros(T, H * dv, dtype=dtype, device="cuda")
    items = dev_i(torch.from_numpy(plan.items)).view(-1)
    tables = dev_i(table[None, :].repeat(len(segs), 1))
    positions = dev_i(torch.cat([torch.arange(s.start, s.start + s.count) for s in segs]))
    tpr, tns = dev_i(torch.from_numpy(plan.tok_part_row)), dev_i(torch.from_numpy(plan.tok_nsplit))
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    gate = dict(gate=gate, gate_per_head=per_head) if gate is not None else {}
    common = dict(nq=H, nkv=G, d=d, page_size=P_, window=window, scale=scale, **gate, **opts)
    if kernel == "simt":
        n = plan.n_small + plan.n_big
        K.attention_simt(q, pool, o, part_acc, part_ml, items, n, n, positions, tables, tpr, dv=dv, **common)
        if plan.part_rows:
            K.attention_combine(part_acc, part_ml, tpr, tns, o, nq=H, d=dv, **gate)
        return o.float().cpu().double().view(T, H, dv), plan
    if plan.n_small:
        counters = torch.zeros(T * G * -(-(H // G) // 16), dtype=torch.int32, device="cuda")
        args = (q, pool, o, part_acc, part_ml, items, plan.n_small, 16, positions, tables, tpr)
        if kernel == "tc":
            K.attention_tma_ext(*args, **common, tok_nsplit=tns, counters=counters, status=status)
        else:
            K.attention_mma_ext(*args, dv=dv, **common, tok_nsplit=tns, counters=counters)
        assert int(counters.abs().sum()) == 0
    if plan.n_big and kernel == "tc":
        K.attention_tc_ext(q, pool, o, items[plan.n_small * 8:], plan.n_big, positions, tables, status=status,
                           part_acc=part_acc, part_ml=part_ml, tok_part_row=tpr, **common)
        if plan.big_split:
            K.attention_combine(part_acc, part_ml, tpr, tns, o, nq=H, d=dv, **gate)
    elif plan.n_big:
        K.attention_mma_ext(q, pool, o, part_acc, part_ml, items[plan.n_small * 8:], plan.n_big, 64, positions, tables, tpr,
                            dv=dv, **common)
    assert int(status) == 0
    return o.float().cpu().double().view(T, H, dv), plan


@pytest.mark.parametrize("H,G,d,dv,P_,size,L", [(6, 3, 24, 40, 16, 21, 150), (1, 1, 20, 20, 8, 1, 60), (4, 2, 64, 64, 16, 96, 420),
                                                (4, 1, 128, 128, 32, 70, 300), (8, 8, 64, 64, 8, 2, 90), (3, 1, 16, 24, 7, 12, 64),
                                                (36, 2, 32, 32, 16, 40, 120), (2, 2, 64, 64, 16, 1150, 1300)])
@pytest.mark.parametrize("dtype,kernel", [(torch.float32, "simt"), (torch.bfloat16, "simt"), (torch.bfloat16, "mma"),
                                          (torch.bfloat16, "tc")])
@pytest.mark.parametrize("biased", [True, False])
def test_attention_at_the_windows_edges(H, G, d, dv, P_, size, L, dtype, kernel, biased):
    """With distance biases, a sink of score 0 and a gate per element ("biased"), or without either and a gate per head:
    one key stands out for the last rows of a portion, of a short portion and of decoded tokens: the oldest position
    inside the window, the one before it, the last row of a page and the first of the next, the row itself.  What the
    cases are for is checked on the plain function: a window one off, no bias and no sink are far from right."""
    from test_rizovik_gpu import Pool, segments_of

    if kernel == "mma" and (d % 8 or dv % 8) or kernel == "tc" and not (d == dv and d in (64, 128)):
        pytest.skip("widths this kernel does not take")
    g = torch.Generator().manual_seed(H * d + L)
    scale = 0.25
    spans = [(L - 41, 30), (L - 11, 3), (L - 8, 1), (L - 7, 2), (L - 5, 1), (L - 4, 4)]
    segs = segments_of(spans)
    T = sum(c for _, c in spans)
    qpos = torch.cat([torch.arange(s, s + c) for s, c in spans])
    gates = torch.randn(T, (H * dv if biased else H) + 3, generator=g)
    gate = gates[:, 2:-1].double()
    gate = torch.sigmoid(gate.view(T, H, dv) if biased else gate[:, :, None])
    slope = P.slopes(H) if biased else None
    for case in ("window_in", "window_out", "page_last", "page_first", "self", "none"):
        q = torch.randn(T, H, d, generator=g)
        k, v = torch.randn(L, G, d, generator=g), torch.randn(L, G, dv, generator=g)
        if case == "none":                      # scores far below the sink: most of the weight goes to it
            q *= 0.02
        for row in (29, 32, 33, T - 1):
            i = int(qpos[row])
            at = {"window_in": max(0, i - size + 1), "window_out": max(0, i - size), "page_last": max(0, i // P_ * P_ - 1),
                  "page_first": i // P_ * P_, "self": i, "none": None}[case]
            for hd in range(0, H, H // G):
                if at is not None:
                    top = 12.0 + (float(slope[hd]) * (i - at) if biased else 0.0)
                    k[at, hd // (H // G)] = q[row, hd] / q[row, hd].norm() * (top / scale / float(q[row, hd].norm()))
        pl = Pool(L, G, d, dv, P_, 0, dtype, seed=3)
        kc, vc = pl.fill(k, v)
        qd = q.to(dtype).cuda()

        def plain(window=size, slope_=slope, sink=biased):
            return P.window_attend(qd.cpu().double(), kc, vc, scale, window, slope=slope_, sink=sink, qpos=qpos) * gate

        ref = plain()
        if case == "window_out" and size < L - 10:
            assert float((plain(window=size + 1) - ref).abs().max()) > 0.05
        if case == "window_in" and size > 1:
            assert float((plain(window=size - 1) - ref).abs().max()) > 0.05
        if case == "none" and biased:
            assert float((plain(sink=False) - ref).abs().max()) > 0.02
            assert size == 1 or float((plain(slope_=None) - ref).abs().max()) > 0.005
        opts = dict(sink=torch.zeros(H, device="cuda"), slopes=slope.float().cuda()) if biased else {}
        for sms in (148, 100000):                # as planned for this GPU, and with as many key splits as there can be
            got, plan = attend(kernel, pl.storage, pl.table, qd.view(T, H * d), segs, H=H, G=G, d=d, dv=dv, P_=P_, window=size,
                               scale=scale, sms=sms, dtype=dtype, gate=gates.cuda()[:, 2:-1], per_head=not biased, **opts)
            close(got, ref, 3e-6 if dtype == torch.float32 else 0.012, f"{case}, {plan.part_rows} partial rows")


@pytest.mark.parametrize("dtype,kernel", [(torch.float32, "simt"), (torch.bfloat16, "mma"), (torch.bfloat16, "tc")])
def test_first_tokens_and_a_bias_over_far_keys(dtype, kernel):
    """No window: a prompt from position 0 (its first tokens share their weight with the sink) and a decoded token behind
    a thousand keys, of which one far back outweighs its bias; key splits carry sink and bias a single time."""
    from test_rizovik_gpu import Pool, segments_of

    g = torch.Generator().manual_seed(2)
    H, G, d, P_, scale, L = 8, 2, 64, 16, 0.25, 1100
    slope = P.slopes(H)
    for spans in ([(0, 40)], [(L - 1, 1)], [(0, 3)], [(L - 200, 200)]):
        segs, T = segments_of(spans), sum(c for _, c in spans)
        qpos = torch.cat([torch.arange(s, s + c) for s, c in spans])
        q, k, v = torch.randn(T, H, d, generator=g), torch.randn(L, G, d, generator=g), torch.randn(L, G, d, generator=g)
        far, hd = 5, H - 1                                       # the last head has the flattest slope
        i = int(qpos[-1])
        if i > 100:
            top = float(slope[hd]) * (i - far) + 14.0
            k[far, G - 1] = q[-1, hd] / q[-1, hd].norm() * (top / scale / float(q[-1, hd].norm()))
        pl = Pool(L, G, d, d, P_, 0, dtype, seed=4)
        kc, vc = pl.fill(k, v)
        qd = q.to(dtype).cuda()
        ref = P.window_attend(qd.cpu().double(), kc, vc, scale, L + 1, slope=slope, sink=True, qpos=qpos)
        if i > 100:
            assert float((ref[-1, hd] - vc[far, G - 1]).abs().max()) < 0.2     # it reaches the output
        for sms in (148, 100000):
            got, plan = attend(kernel, pl.storage, pl.table, qd.view(T, H * d), segs, H=H, G=G, d=d, dv=d, P_=P_, window=0,
                               scale=scale, sms=sms, dtype=dtype, sink=torch.zeros(H, device="cuda"), slopes=slope.float().cuda())
            close(got, ref, 3e-6 if dtype == torch.float32 else 0.012, f"{spans}, {plan.part_rows} partial rows")


@pytest.mark.parametrize("T,n,top,groups,nsplit", [(40, 8, 2, (4, 2), 1), (9, 1, 1, None, 2), (33, 16, 3, (4, 3), 2), (5, 4, 2, (4, 2), 1),
                                                   (70, 40, 35, (2, 2), 1), (21, 12, 4, (2, 1), 3), (17, 64, 6, (8, 3), 2)])
def test_router_by_sigmoid_scores_in_groups(T, n, top, groups, nsplit):
    """Sigmoid scores, choice by score plus correction inside the groups whose two best choice scores sum highest, weights
    without the correction, times a factor and not divided by their sum.  Corrections are large enough to make choice
    scores negative and to let a group with the largest single score lose."""
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(T + n)
    z = torch.randn(nsplit, T, n + 3, generator=g) * 1.5
    corr = torch.randn(n, generator=g) * 0.5 - 0.6
    zd = z.cuda()
    chosen, weights = torch.empty(T, top, dtype=torch.int32, device="cuda"), torch.empty(T, top, device="cuda")
    K.moe_route(Parts(zd if nsplit > 1 else zd[0], nsplit), corr.cuda(), chosen, weights, outputs=n, top=top,
                groups=groups[0] if groups else 1, keep=groups[1] if groups else 1, score="sigmoid", group_two=True,
                normalise=False, factor=1.7)
    w = {"router": torch.eye(n, dtype=torch.float64), "correction": corr.double()}
    r = dict(top=top, scale=1.7, groups=dict(count=groups[0], keep=groups[1]) if groups else None)
    ref_idx, ref_w = P.route(z.double().sum(0)[:, :n], w, "", r)
    assert torch.equal(chosen.cpu().long(), ref_idx)
    close(weights, ref_w, 3e-6, "weights")
    if groups == (4, 2) and n == 8:           # by the largest alone other groups would win somewhere
        best = (torch.sigmoid(z.double().sum(0)[:, :n]) + corr.double()).view(T, 4, 2).max(-1).values
        other = torch.topk(best, 2, -1).indices.sort(-1).values
        mine = torch.stack([torch.unique(row // 2).sum() for row in ref_idx])
        assert bool((mine != other.sum(-1)).any())


@pytest.mark.parametrize("T,W,ff,E,top,shared", [(37, 96, 40, 6, 2, True), (3, 64, 24, 5, 3, False), (300, 128, 64, 4, 2, True), (9, 50, 20, 3, 1, True)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_relu_squared_experts_and_an_ungated_shared_one(T, W, ff, E, top, shared, dtype):
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(T + W)
    h = torch.randn(T, W, generator=g).to(dtype)
    up, down = (torch.randn(E, ff, W, generator=g) * W ** -0.5).to(dtype), (torch.randn(E, W, ff, generator=g) * ff ** -0.5).to(dtype)
    chosen = torch.stack([torch.randperm(E, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    weights = torch.rand(T, top, generator=g)
    sh = torch.randn(2, T, W, generator=g) if shared else None
    ref = sh.double().sum(0) if shared else torch.zeros(T, W, dtype=torch.float64)
    for t in range(T):
        for e, wt in zip(chosen[t].tolist(), weights[t].double()):
            a = P.relu_squared(up[e].double() @ h[t].double())
            ref[t] += wt * (down[e].double() @ (a.to(dtype).double() if dtype == torch.bfloat16 else a))
    pairs = T * top
    plan = torch.empty(K.moe_plan_words(pairs, E), dtype=torch.int32, device="cuda")
    K.moe_plan(chosen.cuda(), plan, experts=E)
    act, y = torch.full((pairs, ff), float("nan"), dtype=dtype, device="cuda"), torch.full((pairs, W), float("nan"), device="cuda")
    K.moe_linear(h.cuda(), plan, up.cuda(), act, pairs=pairs, experts=E, gather=True, act="relu2")
    K.moe_linear(act, plan, down.cuda(), y, pairs=pairs, experts=E, gather=False)
    out = torch.empty(T, W, device="cuda")
    K.moe_combine(y, plan, chosen.cuda(), weights.cuda(), h.cuda(), out, experts=E, shared=Parts(sh.cuda(), 2) if shared else None)
    close(out, ref, 1e-5 if dtype == torch.float32 else 0.01, "routed sum")


@pytest.mark.parametrize("act,fn", [("gelu", P.gelu), ("relu2", P.relu_squared)])
@pytest.mark.parametrize("M,N,Kd", [(300, 96, 64), (1000, 520, 136), (2048, 2048, 256)])
def test_activations_alone_and_in_the_products_epilogue(act, fn, M, N, Kd):
    from mini_hisparse_b200.kernels import api as K

    g = torch.Generator().manual_seed(M)
    x = (torch.randn(M, Kd, generator=g) * 2).to(torch.bfloat16)
    w = (torch.randn(N, Kd, generator=g) * Kd ** -0.5).to(torch.bfloat16)
    z = x.double() @ w.double().T
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    out = torch.empty(M, N, dtype=torch.bfloat16, device="cuda")
    K.gemm_tc_act(x.cuda(), w.cuda(), out, act, status=status, scratch=K.stream_k_scratch("cuda"))
    close(out.float(), fn(z), 0.004)
    assert int(status) == 0
    parts = torch.randn(2, 33, 50, generator=g) * 3
    for n_parts in (1, 2):
        out32 = torch.empty(33, 50, device="cuda")
        pd = parts.cuda()
        K.act_rows(pd if n_parts == 2 else pd[0], out32, act, nsplit=n_parts, split_stride=pd.stride(0))
        close(out32, fn(parts[:n_parts].double().sum(0)), 2e-6)


# ---- the model through the step function ---------------------------------------------------------------------
@pytest.mark.parametrize("name", ["A", "B", "C"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_every_schedule_agrees_with_the_plain_model(models, name, dtype):
    """Whole prompts; most of a prompt and then its tail token by token, three requests side by side (captured graphs; the
    windows pass over decoded tokens); portions of changing size down to two tokens; mixed batches with up to four live
    requests over a pool that holds no more than they need, so that pages and slots are used again (freed pages are
    poisoned).  Every position is compared, with the plain model and with the whole prompt."""
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
        seen[i] = x.detach().float().cpu().clone() + (pending.reduced().cpu() if pending is not None else 0)

    runner.observer = observer
    cache.open("a")
    runner.step([StepEntry("a", toks, [len(toks) - 1])])
    runner.check_status()
    for i in range(len(cfg["layers"])):
        err = row_errors(seen[i], streams[i])
        err = float(err.max() if dtype == "float32" else err.median())       # bfloat16: single rows take another expert
        assert err < (1e-5 if dtype == "float32" else 0.015), f"after layer {i}: {err:.3g}"
    assert torch.equal(seen["final"], seen[len(cfg["layers"]) - 1])


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_far_tokens_through_layers_of_windows(tmp_path, dtype):
    """A request of 900 tokens under windows of 300 and 150 whose keys stand out (large q and k weights against small
    slopes' biases): what the last positions know of far tokens passes window after window, with key splits.  Decoded
    tokens and short portions far into it, every cut against the plain model, whose last logits do move when an early
    token changes."""
    from mini_hisparse_b200 import write_random_model

    cfg = model(120, 128, [layer("attention", sloped(8, 2, 64, 64, 4, 300, temp=(0.5, 100), scale=0.4), dense(256)),
                           layer("attention_2", keyed(4, 2, 32, 290, rot=16, scale=0.5), moe(4, 2, 64, groups=(2, 1), shared=32)),
                           layer("attention", sloped(4, 2, 64, 64, 4, 310, temp=(0.5, 100), scale=0.4, kv_from=0), dense(128)),
                           layer("attention_2", keyed(4, 4, 64, 150, rot=64, scale=0.4), None)])
    write_random_model(cfg, 37, tmp_path, dtype=torch.bfloat16, matrix_std=0.15)
    cfg, w = P.load_folder(tmp_path)
    reqs = requests_for(cfg, [900], seed=70)
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    changed = list(reqs["r0"])
    changed[200] = (changed[200] + 1) % cfg["vocab"]
    assert float(row_errors(P.forward(cfg, w, changed)[-1:].float(), refs["r0"][-1:])) > 10 * F32_ROW
    for steps in (S.whole(reqs), S.tail_one_by_one(reqs, tail=40), S.changing_portions(reqs, sizes=(530, 2, 7, 64, 3, 2, 200))):
        got, stats, pages = run_steps(tmp_path, dtype, steps)
        check_against_plain(got, refs, dtype)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_other_proportions(tmp_path, dtype):
    """Eighteen query heads on one KV head, heads wider than the tensor cores' tiles, values 8 wide, sixteen taps, an odd
    vocabulary, a reader two layers behind another reader, top equal to what the kept groups hold, a layer order that ends
    without a feed-forward."""
    from mini_hisparse_b200 import write_random_model

    cfg = model(257, 120, [
        layer("attention_2", keyed(18, 1, 40, 11, rot=8), moe(9, 3, 24, groups=(3, 1), shared=8)),
        layer("attention", sloped(2, 2, 144, 8, 16, 25), dense(40)),
        layer("attention", sloped(4, 2, 144, 8, 2, 6, kv_from=1), moe(2, 2, 32)),
        layer("attention", sloped(2, 2, 144, 8, 3, 40, temp=(-0.2, 3), kv_from=1), dense(56)),
        layer("attention_2", keyed(2, 2, 136, 17, rot=136, base=20.0), None)])
    write_random_model(cfg, 17, tmp_path, dtype=torch.bfloat16, matrix_std=0.15)
    cfg, w = P.load_folder(tmp_path)
    reqs = requests_for(cfg, [90, 37, 5], seed=33)
    refs = {rid: P.forward(cfg, w, toks).float() for rid, toks in reqs.items()}
    for steps in (S.whole(reqs), S.mixed(reqs, seed=2, tail=15)):
        got, stats, pages = run_steps(tmp_path, dtype, steps)
        check_against_plain(got, refs, dtype)


def test_the_plain_model_is_sensitive_to_what_the_tests_are_for(models):
    """A window one key off, another temperature, rotation or factor of the weights, a group kept more, reversed filters, a
    missing bias, correction or norm: each moves the plain model's logits by far more than the float32 tolerance."""
    folder, cfg, w = models["A"]
    toks = random_tokens(cfg["vocab"], 90, 5)
    right = P.forward(cfg, w, toks)
    rms = float(right.pow(2).mean().sqrt())

    def moved(cfg2=None, w2=None):
        return float((P.forward(cfg2 or cfg, w2 or w, toks) - right).pow(2).mean().sqrt()) / rms

    def mixer(c, i):
        return c["layers"][i]["mixer"]

    changes = [lambda c: mixer(c, 0)["mask"].update(size=22), lambda c: mixer(c, 0)["mask"].update(size=20),
               lambda c: mixer(c, 1)["mask"].update(size=14), lambda c: mixer(c, 2)["mask"].update(size=33),
               lambda c: mixer(c, 3)["mask"].update(size=9), lambda c: mixer(c, 0)["q_temp"].update(every=10),
               lambda c: mixer(c, 3)["q_temp"].update(every=5), lambda c: mixer(c, 0).pop("q_temp"),
               lambda c: mixer(c, 1)["rot"].update(dims=14), lambda c: c["layers"][1]["mlp"]["router"].update(scale=1.0),
               lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=3), lambda c: c["norm"].update(eps=1e-2),
               lambda c: c["layers"][1]["mlp"].pop("shared"), lambda c: c["layers"][5]["mlp"]["router"].update(top=1)]
    for change in changes:
        c = copy.deepcopy(cfg)
        change(c)
        assert moved(c) > 25 * F32_ROW
    for name, fn in (("l0.mix.q.conv", lambda t: t.flip(-1)), ("l0.mix.v.conv", lambda t: t.flip(-1)),
                     ("l1.mix.k.b", lambda t: t * 0), ("l1.mlp.correction", lambda t: t + torch.arange(8) * 0.2),
                     ("embed.norm", lambda t: t * 0 + 1), ("l2.mix.g", lambda t: t * 0)):
        w2 = dict(w)
        w2[name] = fn(w[name])
        assert moved(w2=w2) > 25 * F32_ROW
    original = P.slopes
    P.slopes = lambda heads: original(heads) * 0.9
    try:
        assert moved() > 25 * F32_ROW
    finally:
        P.slopes = original


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_a_slot_used_again(models, dtype):
    """A short prompt, then 260 tokens one by one (many windows and pages long), two requests side by side; then their
    slots and pages serve new requests."""
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


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_engine(models, dtype):
    """Engine.add_request / run: admission, portions under a token budget, decoding, finishing.  float32 tokens equal the
    plain model's; in bfloat16 nearly every token is the plain model's choice for the engine's own history, or loses to it
    by less than rounding (a token whose row took another expert may not be)."""
    from mini_hisparse_b200 import Engine, load_model

    folder, cfg, w = models["A"]
    engine = Engine(load_model(folder, dtype=dtype), num_pages=40, page_size=16, max_requests=3, max_tokens_per_step=48,
                    graph_after=2)
    prompts = requests_for(cfg, [70, 9, 33], seed=80)
    for rid, p in prompts.items():
        engine.add_request(rid, p, max_new_tokens=12)
    out = engine.run()
    engine.cache.assert_invariants()
    near = []
    for rid, p in prompts.items():
        assert len(out[rid]) == 12
        if dtype == "float32":
            assert out[rid] == P.generate(cfg, w, p, 12)
        else:
            seq = list(p)
            for tok in out[rid]:
                logits = P.forward(cfg, w, seq)[-1]
                near.append(float(logits.max() - logits[tok]) < 0.05 * float(logits.abs().max()))
                seq.append(tok)
    assert dtype == "float32" or sum(near) >= 0.8 * len(near)


def test_command_line_demo_with_a_rudutar_config(capsys):
    """`demo --config configs/rudutar-demo.json`: random weights, three requests through Engine and scheduler."""
    from pathlib import Path

    import mini_hisparse_b200
    from mini_hisparse_b200 import cli

    config = Path(mini_hisparse_b200.__file__).parent / "configs" / "rudutar-demo.json"
    assert cli.main(["demo", "--config", str(config), "--dtype", "bfloat16", "--requests", "3", "--prompt-tokens", "70",
                     "--max-new-tokens", "6"]) == 0
    report = json.loads(capsys.readouterr().out)
    assert [r["generated_tokens"] for r in report["requests"].values()] == [6, 6, 6]


def test_trace_run_picks_the_model_by_its_config(models, tmp_path):
    """bin/trace_run on a Rudutar folder: the same program, cache and step function as for every model."""
    folder, cfg, w = models["B"]
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
