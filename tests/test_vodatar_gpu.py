"""Vodatar on the GPU: each new kernel against its plain statement (tests/kernel_refs.py), inputs made so that a far key, a
soft cap, a lost convolution input or a map read in the other's place shows, and the engine (32-bit and bfloat16)
against the plain model (tests/plain/vodatar_plain.py) under every way of cutting and batching the work."""

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kernel_refs as ref
from freetoken_b200.engine.engine import StepEntry
from helpers import make_engine, mixed_schedule, model_folder, replay_cuts, replay_mixed, replay_whole, tokens_for
from plain.vodatar_plain import PlainVodatar
from test_pabavik_gpu import assert_rows, attention_problem, attn_tol, row_error
from tiny_vodatar import ALL, PAGE, VODA_1, VODA_3

from freetoken_b200.engine.attention_plan import build_plan
from freetoken_b200.kernels import ops

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]


def rnd(*shape, dtype=torch.float32, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(DEV)


def tol(dtype, f32=2e-5, bf16=2e-2):
    return dict(rtol=f32, atol=f32) if dtype == torch.float32 else dict(rtol=bf16, atol=bf16)


def segs(lens):
    """``lens``: (q_len, kv_len) per request -> seg_info [S, 4] and slots 1..S on the device."""
    rows, q0 = [], 0
    for i, (q, kv) in enumerate(lens):
        rows.append((q0, q, kv, i))
        q0 += q
    return (torch.tensor(rows, dtype=torch.int32, device=DEV),
            torch.arange(1, len(lens) + 1, dtype=torch.int32, device=DEV), q0)


def cpu(t):
    if isinstance(t, tuple):
        return tuple(cpu(x) for x in t)
    return t.detach().cpu().clone() if isinstance(t, torch.Tensor) else t


# A bfloat16 run may choose another expert where two choice scores lie closer than rounding moves them; with one or two
# experts a token and looped layers that moves the token's row by half its spread and later rows by what attends to it.  So
# bfloat16 rows are held closely up to the first token with such a choice and as a whole by their median; the 32-bit runs,
# which share all host logic, are held strictly everywhere.
NEAR_TIE = 0.01


def check_rows(got, plain, toks, dtype, what, lo=0, want=None):
    want = plain.logits(toks) if want is None else want
    want = want[lo:lo + got.shape[0]]
    if dtype == "float32":
        assert_rows(got, want, dtype, what)
        return
    assert torch.isfinite(got).all(), what
    e = row_error(got.cpu(), want)
    near = (plain.router_gaps(toks) <= NEAR_TIE).double()
    first = int(near.argmax()) if float(near.max()) else len(toks)
    if first > lo:
        assert float(e[: first - lo].max()) < 0.1, f"{what}: {float(e[: first - lo].max()):.3g} before the first near-tie at {first}"
    assert float(e.max()) < 1.5 and float(e.median()) < 0.15, f"{what}: worst {float(e.max()):.3g}, median {float(e.median()):.3g}"


# --------------------------------------------------------------------------- the pass over the stream
SIZES = [(5, 64, 2), (9, 90, 3), (3, 21, 7), (4, 1030, 1), (6, 3072, 8), (2, 6144, 1), (3, 4096, 16), (2, 2560, 20), (2, 60, 5),
         (3, 12288, 2), (1, 1536, 1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,C,groups", SIZES)
def test_stream_step_every_combination_of_its_parts(dtype, T, C, groups):
    k = 3
    y, gate, shared, passed = (rnd(T, C, dtype=dtype, seed=i) for i in (1, 2, 3, 4))
    rows = rnd(T * k, C, dtype=dtype, seed=5)
    pos = torch.randperm(T * k, generator=torch.Generator().manual_seed(6)).to(torch.int32)
    pos[::4] = -1                                     # routes to experts without rows
    pos = pos.view(T, k).to(DEV)
    aux = torch.rand(T, 2, generator=torch.Generator().manual_seed(7)).to(DEV)
    aux[0, 0] = 0.0
    gb, vec = rnd(C, seed=8), rnd(C, seed=9)
    wa, wr = rnd(C, seed=10) * 0.3 + 1.0, rnd(C, seed=11) * 0.3 + 1.0
    picked = torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV)
    for kw in (dict(x=y), dict(x=y, gate=gate), dict(x=y, gate=gate, gate_bias=gb, vec=vec), dict(vec=vec), dict(),
               dict(x=rows, routed=(pos, k, None, None, None), gate=gate, gate_bias=gb),
               dict(x=rows, routed=(pos, k, shared, aux, passed), gate=gate, gate_bias=gb),
               dict(x=rows, routed=(pos, k, shared, None, None)), dict(x=y, gate=gate, gate_bias=gb, rows=picked)):
        n = 2 if "rows" in kw else T
        for what in ("norm", "norm32", "raw"):
            if what == "raw" and "rows" in kw:
                continue
            res = [rnd(T, C, seed=12), rnd(T, C, seed=12).cpu()]
            wide = [torch.full((n, C + 8), 7.0, dtype=dtype, device=d) for d in (DEV, "cpu")]
            out = [torch.zeros(n, C, dtype=dtype, device=d) for d in (DEV, "cpu")]
            f32 = [torch.zeros(n, C, device=d) for d in (DEV, "cpu")]
            for i, fn in enumerate((ops.stream_step, ref.stream_step)):
                mv = (lambda t: t) if i == 0 else cpu
                args = {a: mv(b) for a, b in kw.items()}
                if "x" in kw:
                    args.update(post_weight=mv(wa), post_eps=1e-5)
                if what == "raw":
                    args.update(raw_out=wide[i][:, 4:4 + C])
                else:
                    args.update(pre_weight=mv(wr), pre_eps=1e-6, out=out[i])
                    if what == "norm32":
                        args.update(norm_f32=f32[i])
                fn(res[i], groups=groups, **args)
            name = f"{sorted(kw)} {what}"
            torch.testing.assert_close(res[0].cpu(), res[1], rtol=2e-5, atol=2e-5, msg=lambda m: f"{name}: stream: {m}")
            torch.testing.assert_close(out[0].float().cpu(), out[1].float(), **tol(dtype), msg=lambda m: f"{name}: out: {m}")
            torch.testing.assert_close(f32[0].cpu(), f32[1], rtol=5e-5, atol=5e-5, msg=lambda m: f"{name}: 32-bit: {m}")
            torch.testing.assert_close(wide[0].float().cpu(), wide[1].float(), **tol(dtype), msg=lambda m: f"{name}: raw: {m}")


def test_stream_step_norms_the_stream_in_place():
    for C, groups in ((64, 2), (90, 3)):
        res, want = rnd(5, C, seed=1), rnd(5, C, seed=1).cpu()
        w = rnd(C, seed=2)
        ops.stream_step(res, groups=groups, pre_weight=w, pre_eps=1e-5, norm_f32=res)
        ref.stream_step(want, groups=groups, pre_weight=w.cpu(), pre_eps=1e-5, norm_f32=want)
        torch.testing.assert_close(res.cpu(), want, rtol=1e-5, atol=1e-5)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("C,groups,taps", [(64, 2, 4), (90, 3, 4), (3072, 8, 4), (6144, 2, 4), (64, 1, 1), (96, 4, 2), (3072, 8, 5), (128, 16, 3),
                                           (7, 1, 16), (12288, 2, 4)])
def test_stream_step_convolves_single_tokens_as_conv_act_convolves_portions(dtype, C, groups, taps):
    """Twenty tokens of three requests one by one, some sitting out steps, slots that an earlier owner filled: the
    outputs are those of the whole rows in one conv_act."""
    n_req, T = 3, 20
    x = [rnd(T, C, seed=20 + r) for r in range(n_req)]  # the streams' rows; nothing is added
    w, wr = rnd(C, taps, seed=2, scale=0.5), rnd(C, seed=3) * 0.3 + 1.0
    state = torch.full((n_req + 1, max(taps - 1, 1), C), 9.0, device=DEV) if taps > 1 else None
    w1 = w.clone()
    w1[:, -1] += 1.0
    whole = []
    for r in range(n_req):
        h = torch.zeros(T, C, dtype=dtype, device=DEV)
        ops.stream_step(x[r].clone(), groups=groups, pre_weight=wr, pre_eps=1e-5, out=h)
        info, slots, _ = segs([(T, T)])
        u = torch.zeros(T, C, dtype=dtype, device=DEV)
        ops.conv_act(h, w1, None, None, None if state is None else torch.zeros(2, taps - 1, C, device=DEV), slots, info, 1, u)
        whole.append(u)
    fed, got = [0] * n_req, [[] for _ in range(n_req)]
    step = 0
    while min(fed) < T:
        live = [r for r in range(n_req) if fed[r] < T and not (step % 3 == r and step % 2)]
        step += 1
        if not live:
            continue
        info = torch.tensor([[i, 1, fed[r] + 1, r] for i, r in enumerate(live)], dtype=torch.int32, device=DEV)
        slots = torch.tensor([r + 1 for r in live], dtype=torch.int32, device=DEV)
        res = torch.stack([x[r][fed[r]] for r in live]).contiguous()
        h, u = (torch.zeros(len(live), C, dtype=dtype, device=DEV) for _ in range(2))
        u32 = torch.zeros(len(live), C, device=DEV)
        ops.stream_step(res, groups=groups, pre_weight=wr, pre_eps=1e-5, out=h, conv=(w, state, slots, info, u, u32))
        torch.testing.assert_close(u32, u.float(), rtol=0, atol=0)
        for i, r in enumerate(live):
            got[r].append(u[i].clone())
            fed[r] += 1
    for r in range(n_req):
        torch.testing.assert_close(torch.stack(got[r]).float(), whole[r].float(), **tol(dtype, 2e-5, 2e-2))


def test_stream_step_refuses_what_does_not_fit():
    from freetoken_b200.errors import KernelError

    res = rnd(4, 64)
    with pytest.raises(KernelError):
        ops.stream_step(res, groups=5, pre_weight=rnd(64), pre_eps=1e-5, norm_f32=res)
    with pytest.raises(KernelError):
        ops.stream_step(res, x=rnd(4, 64), post_weight=rnd(32))


# --------------------------------------------------------------------------- two-map heads
def conv_rope_case(dtype, H, G, D, Dv, n_rot, taps, lens, page, seed=0):
    info, slots, T = segs(lens)
    C = (H + G) * 2 * D + G * Dv
    P = -(-max(2 * D, Dv) // 16) * 16
    x = rnd(T, C, dtype=dtype, seed=seed + 1)
    w = rnd(C, taps, seed=seed + 2, scale=0.5)
    longest = max(kv for _, kv in lens)
    ang = torch.arange(longest)[:, None] * 0.37 ** torch.arange(max(n_rot // 2, 1))[None, :]
    table = torch.cat([ang.cos(), ang.sin()], -1).float().to(DEV) if n_rot else None
    n_pages = sum(-(-kv // page) for _, kv in lens) + 1
    slot_map, positions, first = [], [], page
    for q, kv in lens:
        slot_map += [first + p for p in range(kv - q, kv)]
        positions += list(range(kv - q, kv))
        first += -(-kv // page) * page
    st = rnd(len(lens) + 1, max(taps - 1, 1), C, seed=seed + 3) if taps > 1 else None
    for i, (q, kv) in enumerate(lens):  # a request that held fewer tokens than the state has rows: zeros before its start
        if taps > 1 and kv - q < taps - 1:
            st[i + 1, : taps - 1 - (kv - q)] = 0
    return (x, w, st, slots, info, T, P, table, torch.tensor(positions, dtype=torch.int32, device=DEV),
            torch.tensor(slot_map, dtype=torch.int32, device=DEV), n_pages)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv,n_rot,taps,page", [(4, 2, 8, 20, 8, 3, 4), (1, 1, 10, 7, 6, 1, 4), (3, 1, 64, 128, 64, 4, 16),
                                                   (6, 3, 12, 28, 8, 5, 8), (2, 2, 9, 30, 4, 2, 4), (2, 1, 32, 64, 0, 4, 16),
                                                   (1, 1, 5, 11, 2, 16, 4), (48, 8, 64, 128, 64, 4, 16)])
def test_conv_rope_store(dtype, H, G, D, Dv, n_rot, taps, page):
    """Requests that start, requests that go on, single tokens, portions shorter than the taps and longer than a tile; fresh
    pages hold NaN: every column that the attention kernels read of a stored row is written."""
    lens = [(37, 37), (1, 9), (2, 30), (taps, taps + 5), (1, 1), (17, 40), (1, 2)]
    x, w, st, slots, info, T, P, table, positions, smap, n_pages = conv_rope_case(dtype, H, G, D, Dv, n_rot, taps, lens, page)
    smap[5] = -1  # not stored
    res = []
    for dev, fn in ((DEV, ops.conv_rope_store), ("cpu", ref.conv_rope_store)):
        mv = (lambda t: t) if dev == DEV else cpu
        ks, vs = (torch.full((n_pages, G, page, P), float("nan"), dtype=dtype, device=dev) for _ in range(2))
        q = torch.full((T, 2 * H, P), float("nan"), dtype=dtype, device=dev)
        state = None if st is None else mv(st).clone()
        fn(mv(x), mv(w), state, mv(slots), mv(info), len(lens), H, G, 2, D, Dv, n_rot, True, mv(positions), mv(table), q, ks, vs,
           mv(smap))
        res.append((q, ks, vs, state))
    for name, a, b in zip(("q", "keys", "values"), res[0], res[1]):
        torch.testing.assert_close(a.float().cpu(), b.float(), equal_nan=True, **tol(dtype), msg=lambda m: f"{name}: {m}")
    if st is not None:
        torch.testing.assert_close(res[0][3].cpu(), res[1][3], rtol=0, atol=0)
    q = res[0][0]
    assert float(q[:, 0::2, D:].abs().max()) == 0 and float(q[:, 1::2, :D].abs().max()) == 0


@pytest.mark.parametrize("cuts", [[50], [1] * 50, [2, 3, 16, 17, 1, 11], [15, 1, 16, 2, 16]])
def test_conv_rope_store_cut_anywhere_is_the_whole(cuts):
    H, G, D, Dv, n_rot, taps, page = 2, 1, 8, 12, 6, 4, 4
    x, w, _, slots, info, T, P, table, positions, smap, n_pages = conv_rope_case(torch.float32, H, G, D, Dv, n_rot, taps, [(50, 50)], page)
    outs = []
    for parts in ([50], cuts):
        ks, vs = (torch.zeros(n_pages, G, page, P, device=DEV) for _ in range(2))
        q = torch.zeros(T, 2 * H, P, device=DEV)
        state = torch.full((2, taps - 1, x.shape[1]), 7.0, device=DEV)  # the slot's earlier owner left something behind
        i = 0
        for c in parts:
            info, slots, _ = segs([(c, i + c)])
            ops.conv_rope_store(x[i:i + c], w, state, slots, info, 1, H, G, 2, D, Dv, n_rot, True, positions[i:i + c].clone(), table,
                                q[i:i + c], ks, vs, smap[i:i + c].clone())
            i += c
        outs.append((q, ks, vs, state))
        assert i == T
    for a, b in zip(*outs):
        torch.testing.assert_close(a, b, rtol=1e-6, atol=1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,Dv,P", [(5, 3, 20, 32), (7, 2, 128, 128), (1, 1, 7, 32), (3, 4, 64, 64), (2, 3, 256, 256), (9, 2, 8, 16)])
def test_diff_heads(dtype, T, H, Dv, P):
    o = rnd(T, 2 * H, P, dtype=dtype, seed=1)
    lam = torch.tensor([0.37], device=DEV)
    got, want = torch.zeros(T, H, Dv, dtype=dtype, device=DEV), torch.zeros(T, H, Dv, dtype=dtype)
    ops.diff_heads(o, lam, 1e-5, 0.7, got)
    ref.diff_heads(o.cpu(), lam.cpu(), 1e-5, 0.7, want)
    torch.testing.assert_close(got.float().cpu(), want.float(), **tol(dtype))


# --------------------------------------------------------------------------- soft cap inside attention
def run_capped(dtype, Hq, Hkv, D, P, lens, tile, scale, cap, split=False, few=False, problem=None):
    q, ks, vs, bt, seg = problem or attention_problem(dtype, Hq, Hkv, D, P, lens)
    kw = dict(sm_count=4096, min_split_keys=32) if split else dict(sm_count=148)
    if tile >= 128 or few:
        kw["key_tile"] = 128
        if split:
            kw["min_split_keys"] = 128
    plan = build_plan(lens, Hq // Hkv, tile, None, Hkv, **kw)
    items = torch.from_numpy(plan.items).to(DEV)
    po = pm = None
    if plan.n_slots:
        po = torch.full((plan.n_slots, Hkv, tile, D), float("nan"), dtype=torch.float32, device=DEV)
        pm = torch.full((plan.n_slots, Hkv, tile, 2), float("nan"), dtype=torch.float32, device=DEV)
    out, want = torch.full(q.shape, float("nan"), dtype=dtype, device=DEV), torch.empty(q.shape, dtype=dtype, device=DEV)
    ops.paged_attention(q, ks, vs, bt, seg, len(lens), items, plan.n_items, po, pm, out, tile, scale, None, few_rows=few, softcap=cap)
    ref.paged_attention(q, ks, vs, bt, seg, len(lens), items, plan.n_items, None, None, want, tile, scale, None, softcap=cap)
    assert ops.read_status() == 0
    return out, want


# caps: every score small against it, some, none; and one so large that it cannot serve as the maximum
CAPS = [(60.0, 1.0), (30.0, 1.0), (6.0, 2.0), (1.5, 3.0), (200.0, 8.0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap,mult", CAPS)
@pytest.mark.parametrize("Hq,Hkv,D,P,split", [(4, 2, 64, 16, False), (6, 3, 16, 4, True), (12, 1, 128, 16, True), (2, 2, 48, 8, False)])
def test_attention_with_a_soft_cap(dtype, cap, mult, Hq, Hkv, D, P, split):
    lens = [(1, 1), (5, 5), (70, 70), (2, 131), (1, 64), (33, 97), (1, 300)]
    for tile in ([16] if dtype == torch.float32 else [16, 64]):
        out, want = run_capped(dtype, Hq, Hkv, D, P, lens, tile, mult * D ** -0.5, cap, split)
        torch.testing.assert_close(out.float().cpu(), want.float().cpu(), **attn_tol(dtype))


@pytest.mark.parametrize("cap,mult", CAPS)
@pytest.mark.parametrize("form", ["one tile", "two tiles", "few rows"])
@pytest.mark.parametrize("Hq,Hkv,P,split", [(4, 4, 16, False), (12, 2, 16, True), (12, 1, 32, False), (6, 3, 64, True)])
def test_the_tensor_core_kernels_take_the_soft_cap(form, cap, mult, Hq, Hkv, P, split):
    """Heads of 128: long portions, portions behind hundreds of cached tokens, single tokens, tiles cut along the keys; groups
    that do not fill a tile's rows (12 heads: 120 of 128), whose other rows hold anything."""
    few = form == "few rows"
    lens = [(1, 64), (1, 300), (1, 128), (1, 129), (1, 515)] if few else [(300, 300), (130, 700), (1, 64), (128, 128), (2, 515)]
    tile = 16 if few else 256 if form == "two tiles" else 128
    ops.variant_counts(reset=True)
    out, want = run_capped(torch.bfloat16, Hq, Hkv, 128, P, lens, tile, mult * 128 ** -0.5, cap, split, few)
    assert sum(n for k, n in ops.variant_counts().items() if "tcgen05" in k and "soft cap" in k) == 1
    torch.testing.assert_close(out.float().cpu(), want.float().cpu(), **attn_tol(torch.bfloat16))


@pytest.mark.parametrize("form", ["float32", "mma 16", "mma 64", "few rows", "one tile", "two tiles"])
def test_a_far_key_that_stands_out_is_held_down_by_the_cap(form):
    """One key 250 places back scores 40 against 0 for all others: without a cap it takes all the weight, with a cap of 3 its
    score is 3 tanh(40 / 3), so it gets e^3 against 1 each for the other keys."""
    dtype = torch.float32 if form == "float32" else torch.bfloat16
    Hq, Hkv, D, P = 2, 1, 128, 16
    single = form not in ("one tile", "two tiles", "mma 64")
    lens = [(1, 300)] if single else [(130, 300)]
    q, ks, vs, bt, seg = attention_problem(dtype, Hq, Hkv, D, P, lens, seed=4)
    last = 299
    far = last - 250
    ks.nan_to_num_(0.0).zero_()
    page = int(bt[1, far // P])
    ks[page, 0, far % P, 0] = 10.0
    q[:] = 0
    q[:, :, 0] = 4.0
    tile, few = {"float32": (16, False), "mma 16": (16, False), "mma 64": (64, False), "few rows": (16, True), "one tile": (128, False),
                 "two tiles": (256, False)}[form]
    out, want = run_capped(dtype, Hq, Hkv, D, P, lens, tile, 1.0, 3.0, False, few, (q, ks, vs, bt, seg))
    torch.testing.assert_close(out.float().cpu(), want.float().cpu(), **attn_tol(dtype))
    v = torch.stack([vs[int(bt[1, j // P]), 0, j % P] for j in range(300)]).float().cpu()
    e = torch.ones(300)
    e[far] = torch.exp(3.0 * torch.tanh(torch.tensor(40.0 / 3.0)))
    torch.testing.assert_close(out[-1, 0].float().cpu(), (e[:, None] * v).sum(0) / e.sum(), rtol=2e-2, atol=5e-3)


# --------------------------------------------------------------------------- routing with identity experts
@pytest.mark.parametrize("T,E,n_id,k,extra", [(1, 8, 2, 2, 1), (7, 6, 3, 4, 1), (32, 64, 8, 8, 1), (5, 4, 0, 2, 1), (3, 4, 4, 3, 0), (40, 200, 56, 6, 1)])
def test_routing_with_identity_experts_and_an_extra_logit(T, E, n_id, k, extra):
    C, H = E + n_id, 64
    x = rnd(T, H, seed=1)
    w = rnd(C + extra, H, seed=2, scale=H ** -0.5)
    corr = rnd(C, seed=3, scale=0.1)
    shapes = dict(ids=((T, k), torch.int32), wts=((T, k), torch.float32), aux=((T, 2), torch.float32))
    mk = lambda d: {n: torch.zeros(*s, dtype=t, device=d) for n, (s, t) in shapes.items()}  # noqa: E731
    want = mk("cpu")
    logits = x.cpu() @ w.cpu().T
    ref.router_topk(logits, corr.cpu(), k, "softmax", 1.0, want["ids"], want["wts"], n_extra=extra, n_real=E, aux=want["aux"])
    got = mk(DEV)
    parts = torch.cat([logits * 0.75, logits * 0.25], -1).to(DEV).contiguous()
    padded = torch.cat([torch.nn.functional.pad(logits * f, (0, 3), value=1e9) for f in (0.75, 0.25)], -1).to(DEV).contiguous()
    for n_parts, lg, pad in ((1, logits.to(DEV), 0), (2, parts, 0), (2, padded, 3)):
        ops.router_topk(lg, corr, k, "softmax", 1.0, got["ids"], got["wts"], n_parts=n_parts, n_extra=extra, n_real=E, aux=got["aux"],
                        n_pad=pad)
        torch.testing.assert_close(got["ids"].cpu(), want["ids"], rtol=0, atol=0)
        torch.testing.assert_close(got["wts"].cpu(), want["wts"], rtol=1e-5, atol=1e-6)
        torch.testing.assert_close(got["aux"].cpu(), want["aux"], rtol=1e-5, atol=1e-6)
    if not ops.moe_route_fits(T, H, C, k):
        return
    got = mk(DEV)
    i32 = lambda n, d: torch.zeros(n, dtype=torch.int32, device=d)  # noqa: E731
    sort_g = (i32(E, DEV), i32(E + 1, DEV), i32(T * k, DEV), i32(T * k, DEV))
    sort_w = (i32(E, "cpu"), i32(E + 1, "cpu"), i32(T * k, "cpu"), i32(T * k, "cpu"))
    lg = torch.zeros(T, C + extra, device=DEV)
    ops.moe_route(x, w, corr, k, "softmax", 1.0, lg, got["ids"], got["wts"], *sort_g, n_extra=extra, n_real=E, aux=got["aux"])
    ref.moe_permute(want["ids"], E, *sort_w)
    torch.testing.assert_close(got["ids"].cpu(), want["ids"], rtol=0, atol=0)
    torch.testing.assert_close(got["aux"].cpu(), want["aux"], rtol=1e-4, atol=1e-5)
    for n, a, b in zip(("counts", "offsets"), sort_g, sort_w):
        torch.testing.assert_close(a.cpu(), b, rtol=0, atol=0, msg=n)
    torch.testing.assert_close(sort_g[3].cpu(), sort_w[3], rtol=0, atol=0)
    n_live = int(sort_w[1][-1])
    torch.testing.assert_close(sort_g[2].cpu()[:n_live], sort_w[2][:n_live], rtol=0, atol=0)
    ops.moe_permute(got["ids"], E, *sort_g)  # the sort of long steps gives identity routes no place either
    torch.testing.assert_close(sort_g[3].cpu(), sort_w[3], rtol=0, atol=0)


@pytest.mark.parametrize("dtype", DTYPES)
def test_moe_combine_with_passed_rows_and_a_weighted_shared_part(dtype):
    T, k, C = 7, 3, 90
    y, shared, passed = rnd(T * k, C, dtype=dtype, seed=1), rnd(T, C, dtype=dtype, seed=2), rnd(T, C, dtype=dtype, seed=3)
    pos = torch.randperm(T * k, generator=torch.Generator().manual_seed(4)).to(torch.int32)
    pos[::5] = -1
    pos = pos.to(DEV)
    aux = torch.rand(T, 2, generator=torch.Generator().manual_seed(5)).to(DEV)
    got, want = torch.zeros(T, C, dtype=dtype, device=DEV), torch.zeros(T, C, dtype=dtype)
    ops.moe_combine(y, pos, T, k, shared, got, aux=aux, passed=passed)
    ref.moe_combine(y.cpu(), pos.cpu(), T, k, shared.cpu(), want, aux=aux.cpu(), passed=passed.cpu())
    torch.testing.assert_close(got.float().cpu(), want.float(), **tol(dtype))


# --------------------------------------------------------------------------- the engine against the plain model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["V1", "V2", "V3", "V4"])
def test_cuts_and_batches_agree_with_the_plain_model(name, dtype, tmp_path_factory):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainVodatar(folder)
    eng = make_engine(folder, dtype, DEV, 16 if name == "V3" else PAGE, pages=40)
    toks = tokens_for(plain.vocab, 70, 11)
    want = plain.logits(toks)
    check_rows(replay_whole(eng, "w", toks), plain, toks, dtype, "whole", want=want)
    check_rows(replay_cuts(eng, "d", toks, [38]), plain, toks, dtype, "last 32 one by one", want=want)
    check_rows(replay_cuts(eng, "c", toks, [7, 2, 13, 2, 5, 3, 2, 11, 2]), plain, toks, dtype, "portions", want=want)
    check_rows(replay_cuts(eng, "one", toks[:24], []), plain, toks, dtype, "one by one from the first token", want=want)
    eng.cache.check()
    eng.check_kernels()
    assert all(g.pool.free_count == g.pool.num_pages for g in eng.cache.paged)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["V1", "V4"])
def test_mixed_steps_with_few_pages_and_slots(name, dtype, tmp_path_factory):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainVodatar(folder)
    lengths = {"r0": 45, "r1": 60, "r2": 38, "r3": 52, "r4": 41, "r5": 47}
    seqs = {r: tokens_for(plain.vocab, n, i) for i, (r, n) in enumerate(lengths.items())}
    eng = make_engine(folder, dtype, DEV, PAGE, pages=4 * (-(-64 // PAGE)))
    got = replay_mixed(eng, seqs, mixed_schedule(lengths, seed=3))
    for r, toks in seqs.items():
        check_rows(got[r], plain, toks, dtype, r)
    for g in eng.cache.paged:
        assert g.pool.handed_out > g.pool.num_pages, "the trace was meant to use pages again"
    assert eng.cache.slots.free_count == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["V1", "V3"])
def test_long_prompt_long_decoding_and_recorded_steps(name, dtype, tmp_path_factory):
    """Hundreds of tokens across many pages, a hundred tokens one by one (recorded into a CUDA graph at the first), and a
    long step in between."""
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainVodatar(folder)
    toks = tokens_for(plain.vocab, 300, 3)
    want = plain.logits(toks)
    eng = make_engine(folder, dtype, DEV, 16, pages=64, max_step=512)
    check_rows(replay_whole(eng, "w", toks), plain, toks, dtype, "whole", want=want)
    check_rows(replay_cuts(eng, "d", toks, [200]), plain, toks, dtype, "a hundred tokens one by one", want=want)
    assert eng.graphs, "the decode steps were meant to be recorded"
    check_rows(replay_cuts(eng, "c", toks, [63, 2, 64, 65, 17, 2, 33] + [1] * 20 + [30, 2]), plain, toks, dtype, "portions", want=want)
    other = tokens_for(plain.vocab, 130, 5)
    got = [eng.step([StepEntry("a", toks[:3], [0, 1, 2])]).logits.float().cpu().clone()]
    for i in range(3, 12):
        got.append(eng.step([StepEntry("a", toks[i:i + 1], [0])]).logits.float().cpu().clone())
    long = eng.step([StepEntry("b", other, list(range(len(other))))]).logits.float().cpu().clone()
    for i in range(12, 40):
        got.append(eng.step([StepEntry("a", toks[i:i + 1], [0])]).logits.float().cpu().clone())
    check_rows(long, plain, other, dtype, "the long step")
    check_rows(torch.cat(got), plain, toks, dtype, "decode steps before and after it", want=want)
    eng.check_kernels()


def test_heads_of_128_run_the_tensor_core_attention(tmp_path_factory):
    folder = model_folder(tmp_path_factory.getbasetemp(), "V3", VODA_3)
    plain = PlainVodatar(folder)
    toks = tokens_for(plain.vocab, 300, 9)
    want = plain.logits(toks)
    eng = make_engine(folder, "bfloat16", DEV, 16, pages=96, max_step=512)
    ops.variant_counts(reset=True)
    check_rows(replay_whole(eng, "w", toks), plain, toks, "bfloat16", "whole", want=want)
    forms = ops.variant_counts()
    assert any("tcgen05" in k and "soft cap" in k for k in forms) and any(k == "attention: tcgen05, 128-row query tiles" for k in forms), forms
    check_rows(replay_cuts(eng, "c", toks, [150, 130, 2]), plain, toks, "bfloat16", "portions, the rest one by one", want=want)
    assert ops.variant_counts().get("attention: tcgen05, tiles of at most 16 rows, soft cap", 0) > 0
    others = {f"o{i}": tokens_for(plain.vocab, 20 + i, 20 + i) for i in range(3)}
    for r, t in others.items():  # three requests that decode beside a long portion
        eng.step([StepEntry(r, t[:-1], [])])
    out = eng.step([StepEntry("long", toks[:200], list(range(200)))] + [StepEntry(r, t[-1:], [0]) for r, t in others.items()])
    check_rows(out.logits[:200].float().cpu(), plain, toks, "bfloat16", "a long portion beside single tokens", want=want)
    for i, (r, t) in enumerate(others.items()):
        assert float(row_error(out.logits[200 + i:201 + i].float().cpu(), plain.logits(t)[-1:]).max()) < 1.5, r
    eng.check_kernels()


REAL_LAYERS = {  # layers of the size of a real model's (no test of the tiny configurations reaches these kernel forms)
    "architecture": "Vodatar", "vocab": 8192, "width": 2048, "norm": {"eps": 1e-6, "groups": 8}, "residual_mult": 0.7,
    "canon": {"taps": 4}, "loop": {"start": 1, "stop": 2, "times": 2},
    "layers": [
        {"type": "attention", "mixer": {"heads": 24, "kv_heads": 4, "dim": 64, "vdim": 128, "conv": 4, "scale": 0.125, "softcap": 25.0,
                                        "diff": 0.35, "rot": {"dims": 64, "base": 500000.0}},
         "mlp": {"kind": "moe", "expert": {"ff": 768}, "router": {"experts": 24, "identity": 3, "top": 4}, "shared": {"ff": 1024}}},
        {"type": "latent_attention", "mixer": {"heads": 16, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 64, "scale": 192 ** -0.5,
                                               "rot": {"dims": 64, "base": 500000.0, "scaling": {
                                                   "factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}, "mlp": None},
    ]}


def test_layers_of_real_sizes_agree_across_cuts_and_dtypes():
    """Heads of 128, long portions: the attention kernels' tcgen05 forms, expert products on the tensor cores with identity
    routes among them, rows of the stream in registers.  No plain model at these sizes: the 32-bit engine is compared
    with itself across cuts, the bfloat16 engine with it."""
    from freetoken_b200.config.engine_config import EngineConfig
    from freetoken_b200.engine.engine import Engine

    toks = tokens_for(REAL_LAYERS["vocab"], 600, 4)
    seen = sorted(set(range(0, 600, 7)) | set(range(560, 600)))

    def rows(eng, rid, cuts):
        got, i, cuts = {}, 0, list(cuts)
        while i < len(toks):
            c = min(cuts.pop(0) if cuts else 1, len(toks) - i)
            want = [p - i for p in seen if i <= p < i + c]
            out = eng.step([StepEntry(rid, toks[i:i + c], want)])
            for j, w in enumerate(want):
                got[w + i] = out.logits[j].float().cpu().clone()
            i += c
        eng.close(rid)
        return torch.stack([got[p] for p in seen])

    res = {}
    for dtype in ("float32", "bfloat16"):
        eng = Engine(EngineConfig(model_path="", dtype=dtype, use_dummy_weight=True, seed=3, page_size=16, max_running_req=4,
                                  num_page_override=100, max_seq_len_override=1024, max_extend_tokens=640, max_step_tokens=640,
                                  check_cache=True), raw_config=REAL_LAYERS)
        ops.variant_counts(reset=True)
        res[dtype, "whole"] = rows(eng, "w", [600])
        if dtype == "bfloat16":
            forms = ops.variant_counts()
            assert sum(n for k, n in forms.items() if "tcgen05" in k and "soft cap" in k) == 1, forms
            assert sum(n for k, n in forms.items() if k.startswith("expert") and "tcgen05" in k) == 2, forms
        res[dtype, "cuts"] = rows(eng, "c", [300, 256, 2, 7])
        eng.check_kernels()
        del eng
        torch.cuda.empty_cache()
    assert torch.isfinite(res["float32", "whole"]).all()
    assert float(row_error(res["float32", "cuts"], res["float32", "whole"]).max()) < 1e-4
    for kind in ("whole", "cuts"):
        e = row_error(res["bfloat16", kind], res["float32", "whole"])
        assert float(e.median()) < 0.03 and float((e > 0.1).double().mean()) < 0.2, (kind, e.sort().values[-20:])


def test_greedy_generation_through_the_scheduler(tmp_path_factory):
    from freetoken_b200 import LLM, SamplingParams

    folder = model_folder(tmp_path_factory.getbasetemp(), "V1", VODA_1)
    plain = PlainVodatar(folder)
    prompts = [[5, 17, 3, 150, 41], [9, 8, 7, 6, 5, 4, 3, 2, 1, 0, 11, 12], [199]]
    for dtype in ("float32", "bfloat16"):
        llm = LLM(folder, dtype=dtype, device=DEV, page_size=4, num_page_override=48, max_step_tokens=8,
                  max_extend_tokens=8, max_running_req=2)  # three prompts on two request slots, in portions of eight
        outs = llm.generate(prompts, SamplingParams(max_tokens=10))
        for p, o in zip(prompts, outs):
            toks = list(p)
            assert len(o["token_ids"]) == 10
            for got in o["token_ids"]:
                logits = plain.logits(toks)[-1]
                top2 = torch.topk(logits, 2).values
                if dtype == "float32" or float(top2[0] - top2[1]) > 0.3:
                    assert got == int(torch.argmax(logits)), (dtype, p, o)
                toks.append(got)


def test_the_replay_tool_runs_the_design(tmp_path_factory, tmp_path):
    folder = model_folder(tmp_path_factory.getbasetemp(), "V4", ALL["V4"])
    plain = PlainVodatar(folder)
    a, b = tokens_for(plain.vocab, 30, 1), tokens_for(plain.vocab, 9, 2)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": a[20:21], "want": [0]}, {"id": "b", "tokens": b[2:], "want": [6]}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[21:], "want": [8]}], "end": ["a"]},
    ]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        p = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", folder, "--dtype", dtype,
                            "--out", str(out), "--max-tokens", "128"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=600)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
        la, lb = plain.logits(a), plain.logits(b)
        got = [np.fromfile(out / f"{i}.f32", dtype="<f4").reshape(-1, plain.vocab) for i in range(3)]
        for i, rows in enumerate((la[[0, 19]], torch.stack([la[20], lb[8]]), la[[29]])):
            e = row_error(torch.from_numpy(got[i]), rows)
            assert float(e.max()) < (1e-4 if dtype == "float32" else 1.0), (dtype, i, e)
