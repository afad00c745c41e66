"""Gizulorn on the GPU: each new kernel path against its plain statement (tests/kernel_refs.py), inputs made so that a kept
first token, a window's edge, a sink, a far key or a lost state shows, and the engine (32-bit and bfloat16) against the
plain model (tests/plain/gizulorn_plain.py) under every way of cutting and batching the work."""

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
from plain.gizulorn_plain import PlainGizulorn
from test_pabavik_gpu import assert_rows, attention_problem, attn_tol, row_error, run_attention
from test_vodatar_gpu import cpu, rnd, segs, tol
from tiny_gizulorn import ALL, GIZU_1, GIZU_3, PAGE

from freetoken_b200.errors import KernelError
from freetoken_b200.kernels import ops
from freetoken_b200.parts.gla import chunk_list

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
DTYPES = [torch.float32, torch.bfloat16]
NEAR_TIE = 0.01  # softmax scores (or group scores) that lie closer than bfloat16 rounding may move them


def check_rows(got, plain, toks, dtype, what, lo=0, want=None):
    """32-bit runs strictly everywhere.  bfloat16 runs (measured: most rows within 0.005 to 0.02) closely up to the first token
    with a near tie in a router, from where on another expert may be as right, and as a whole by their median.  A recurrent
    head's output is divided by its own size: where it nearly vanishes (a first token whose query and key are almost at
    right angles, say) rounding turns it round, so a few rows may lie farther off."""
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
        sure = e[: first - lo]
        assert float(sure.max()) < 0.5 and int((sure > 0.1).sum()) <= max(1, sure.numel() // 20), \
            f"{what}: {int((sure > 0.1).sum())} rows up to {float(sure.max()):.3g} before the first near-tie at {first}"
    assert float(e.max()) < 1.5 and float(e.median()) < 0.15, f"{what}: worst {float(e.max()):.3g}, median {float(e.median()):.3g}"


# --------------------------------------------------------------------------- attention: a window that keeps first tokens
def hide_the_passed(problem, window, keep, P):
    """NaN in every cached row that no query of the step can see (its page may have gone back to the pool)."""
    q, ks, vs, bt, seg = problem
    for q_start, q_len, kv_len, row in seg.tolist():
        for j in range(keep, max(keep, kv_len - q_len - window + 1)):
            ks[int(bt[row, j // P]), :, j % P] = float("nan")
            vs[int(bt[row, j // P]), :, j % P] = float("nan")
    return problem


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,Hkv,D,P,window,keep", [(4, 2, 16, 4, 9, 3), (6, 6, 32, 8, 40, 1), (8, 1, 48, 4, 1, 70), (12, 2, 128, 16, 200, 64),
                                                    (6, 3, 96, 16, 64, 65), (4, 4, 64, 16, 33, 150), (2, 1, 256, 16, 5, 7)])
def test_attention_with_kept_first_tokens(dtype, Hq, Hkv, D, P, window, keep):
    lens = [(1, 1), (5, 5), (70, 70), (2, 131), (1, 64), (33, 297), (1, 300), (keep, keep), (3, keep + window), (3, keep + window + 3)]
    tile = 64 if dtype == torch.bfloat16 else 16
    sink = rnd(Hq, seed=9)
    for s in (sink, None):
        for force in (False, True):
            problem = hide_the_passed(attention_problem(dtype, Hq, Hkv, D, P, lens, seed=3), window, keep, P)
            out, want, _ = run_attention(dtype, Hq, Hkv, D, P, lens, tile, window, s, force_split=force, problem=problem, keep_first=keep)
            torch.testing.assert_close(out.float(), want.float(), **attn_tol(dtype))
    dec = [(1, 1), (1, 17), (1, 64), (1, 65), (1, 333), (1, 128), (1, keep + window), (1, keep + window + 1), (1, 700)]
    for fixed in (None, 1, 5):
        problem = hide_the_passed(attention_problem(dtype, Hq, Hkv, D, P, dec, seed=3), window, keep, P)
        out, want, _ = run_attention(dtype, Hq, Hkv, D, P, dec, 16, window, sink, fixed_splits=fixed, problem=problem, keep_first=keep)
        torch.testing.assert_close(out.float(), want.float(), **attn_tol(dtype))


@pytest.mark.parametrize("Hq,Hkv,P,window,keep", [(12, 2, 16, 200, 4), (4, 4, 32, 37, 128), (16, 1, 16, 128, 129), (6, 2, 48, 1, 1),
                                                  (8, 2, 16, 1000, 20), (6, 2, 64, 5, 300)])
def test_kept_first_tokens_on_the_tensor_core_kernel(Hq, Hkv, P, window, keep):
    """Pieces that jump from the kept tokens' key tiles to the window's, rows between them that hold NaN, pages that do not
    divide a key tile, tiles split along the keys, single tokens."""
    sink = rnd(Hq, seed=9)
    for lens, kw in (([(300, 300)], {}), ([(128, 128), (1, 40), (200, 717), (3, 3), (1, 1300)], {}), ([(256, 1900)], dict(force_split=True)),
                     ([(130, 1000)], {}), ([(1, 700), (1, 64), (1, 129), (1, 1500)], dict(fixed_splits=4))):
        for s in (sink, None):
            problem = hide_the_passed(attention_problem(torch.bfloat16, Hq, Hkv, 128, P, lens, seed=6), window, keep, P)
            ops.variant_counts(reset=True)
            out, want, _ = run_attention(torch.bfloat16, Hq, Hkv, 128, P, lens, 128, window, s, problem=problem, keep_first=keep, **kw)
            assert ops.variant_counts().get("attention: tcgen05, 128-row query tiles, window or sink", 0) == 1
            torch.testing.assert_close(out.float(), want.float(), **attn_tol(torch.bfloat16))
    assert ops.read_status() == 0


@pytest.mark.parametrize("form", ["float32", "mma 16", "mma 64", "tcgen05"])
@pytest.mark.parametrize("window,keep", [(40, 4), (17, 65), (64, 16), (1, 3), (130, 128)])
def test_a_key_at_every_edge_of_the_window_and_of_the_kept_tokens(form, window, keep):
    """One key points where the last query points, twenty times as long.  It is seen at distance window - 1 and as the last kept
    token, and not at distance window or right behind the kept ones, in portions and as a single token, whole and split."""
    dtype = torch.float32 if form == "float32" else torch.bfloat16
    Hq, Hkv, D, P = 4, 2, 128 if form == "tcgen05" else 32, 16
    tile = {"float32": 16, "mma 16": 16, "mma 64": 64, "tcgen05": 128}[form]
    lens = [(1, 390), (1, 401)] if form in ("mma 16", "float32") else [(40, 390), (1, 401)]
    for place, seen in (("inside", True), ("outside", False), ("last kept", True), ("first not kept", False), ("first", True)):
        q, ks, vs, bt, seg = attention_problem(dtype, Hq, Hkv, D, P, lens, seed=4, scale_k=0.3)
        q = q.clone()
        marks = []
        for q_start, q_len, kv_len, row in seg.tolist():
            x = q[q_start + q_len - 1].view(Hkv, Hq // Hkv, D)
            x[:] = x[:, :1] * 3  # all heads of a group ask the same
            j = {"inside": kv_len - window, "outside": kv_len - 1 - window, "last kept": keep - 1, "first not kept": keep, "first": 0}[place]
            last = x[:, 0].float()
            ks[int(bt[row, j // P]), :, j % P] = (20.0 * last / last.norm(dim=-1, keepdim=True)).to(dtype)
            marks.append((q_start + q_len - 1, vs[int(bt[row, j // P]), :, j % P].float()))
        for force in (False, True):
            out, want, _ = run_attention(dtype, Hq, Hkv, D, P, lens, tile, window, rnd(Hq, seed=2), force_split=force,
                                         problem=(q, ks, vs, bt, seg), scale=1.0, keep_first=keep)
            torch.testing.assert_close(out.float(), want.float(), **attn_tol(dtype))
            for t, val in marks:
                got = out[t].float().view(Hkv, Hq // Hkv, D)
                close = float((got - val[:, None, :]).abs().max()) < 0.1 * float(val.abs().max())
                assert close == seen, (place, window, keep, force)


def test_kept_tokens_need_a_window():
    q, ks, vs, bt, seg = attention_problem(torch.float32, 2, 1, 16, 4, [(1, 9)])
    items = torch.zeros(1, 8, dtype=torch.int32, device=DEV)
    with pytest.raises(KernelError):
        ops.paged_attention(q, ks, vs, bt, seg, 1, items, 1, None, None, torch.empty_like(q), 16, 1.0, None, keep_first=3)
    with pytest.raises(KernelError):
        ops.paged_attention(q, ks, vs, bt, seg, 1, items, 1, None, None, torch.empty_like(q), 16, 1.0, 5, keep_first=3, softcap=9.0)


# --------------------------------------------------------------------------- rotation of neighbours on the way to the cache
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,Dp,n_rot,H,G,off", [(64, 64, 64, 4, 2, 0), (128, 128, 64, 3, 1, 8), (24, 32, 8, 2, 2, 5), (10, 16, 6, 1, 1, 3),
                                                (256, 256, 256, 2, 1, 0), (64, 80, 48, 2, 1, 0)])
@pytest.mark.parametrize("neighbours", [True, False])
def test_norm_rope_store_both_pairings(dtype, D, Dp, n_rot, H, G, off, neighbours):
    T, P = 9, 4
    wide = rnd(T, off + (H + G) * D + 7, dtype=dtype, seed=1)
    x = wide[:, off: off + (H + G) * D]
    ang = torch.arange(50)[:, None] * 0.37 ** torch.arange(n_rot // 2)[None, :]
    table = torch.cat([ang.cos(), ang.sin()], -1).float().to(DEV)
    pos = torch.tensor([0, 1, 2, 5, 9, 30, 31, 49, 7], dtype=torch.int32, device=DEV)
    smap = torch.tensor([4, 5, -1, 8, 9, 10, 19, 18, 6], dtype=torch.int32, device=DEV)
    res = []
    for dev, fn in ((DEV, ops.norm_rope_store), ("cpu", ref.norm_rope_store)):
        mv = (lambda t: t) if dev == DEV else cpu
        q = torch.full((T, H, Dp), float("nan"), dtype=dtype, device=dev)
        slab = torch.full((5, G, P, Dp), float("nan"), dtype=dtype, device=dev)
        fn(mv(x), D, n_rot, mv(pos), mv(table), 1e-6, False,
           [dict(first_head=0, n_heads=H, norm_weight=None, rotate=True, dense_out=q, dst_head_dim=Dp),
            dict(first_head=H, n_heads=G, norm_weight=None, rotate=True, slab=slab, slot_map=mv(smap), dst_head_dim=Dp)],
           neighbours=neighbours)
        res.append((q, slab))
    for a, b in zip(*res):
        torch.testing.assert_close(a.float().cpu(), b.float(), equal_nan=True, **tol(dtype))


# --------------------------------------------------------------------------- the delta rule with a decay per key channel
def delta_case(dtype, H, G, D, Dv, T, seed=0):
    rows = rnd(T, 2 * G * D + H * Dv + H + 3, dtype=dtype, seed=seed + 1)
    z = rnd(T, H * D, seed=seed + 2, scale=2.0)
    return (rows[:, :G * D], rows[:, G * D:2 * G * D], rows[:, 2 * G * D:2 * G * D + H * Dv], rows[:, -H - 3:-3], z,
            rnd(H, seed=seed + 3, scale=0.5) - 1.0, rnd(H * D, seed=seed + 4))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 4, 32, 64), (4, 2, 16, 24), (3, 1, 40, 10), (2, 2, 8, 33), (1, 1, 128, 128), (6, 3, 64, 128),
                                      (2, 1, 256, 64), (1, 1, 5, 3), (40, 20, 128, 128), (2, 2, 13, 7)])
def test_the_delta_rule_with_a_decay_per_channel(dtype, H, G, D, Dv):
    """Fresh and continued requests, even and odd numbers of tokens, single tokens, more than a staged batch; steps in which
    some request brings several tokens and steps of single tokens (which turn logits into decays themselves)."""
    for lens in ([(45, 45), (1, 40), (17, 100), (2, 2), (1, 1), (32, 64)], [(1, 1), (1, 40), (1, 7)]):
        info, slots, T = segs(lens)
        q, k, v, b, z, a_log, dt_bias = delta_case(dtype, H, G, D, Dv, T)
        state = rnd(len(lens) + 1, H, Dv, D, seed=9, scale=0.3)
        st_a, st_b = state.clone(), state.cpu().clone()
        got, want = torch.full((T, H, Dv), float("nan"), device=DEV), torch.zeros(T, H, Dv)
        ops.delta_scan(q, k, v, b, None, a_log, dt_bias, D ** -0.5, 1e-6, st_a, slots, info, len(lens), got, z=z.clone())
        ref.delta_scan(q.cpu(), k.cpu(), v.cpu(), b.cpu(), None, a_log.cpu(), dt_bias.cpu(), D ** -0.5, 1e-6, st_b, slots.cpu(),
                       info.cpu(), len(lens), want, z=z.cpu())
        torch.testing.assert_close(got.cpu(), want, rtol=2e-4, atol=2e-5)
        torch.testing.assert_close(st_a.cpu()[1:], st_b[1:], rtol=2e-4, atol=2e-5)
        assert torch.equal(st_a[0], state[0])


@pytest.mark.parametrize("D", [16, 64, 128])
def test_equal_channel_decays_are_the_decay_per_head(D):
    H, G, Dv = 4, 2, 32
    lens = [(37, 37), (1, 9)]
    info, slots, T = segs(lens)
    q, k, v, b, _, a_log, _ = delta_case(torch.float32, H, G, D, Dv, T)
    a, dt_bias = rnd(T, H, seed=21), rnd(H, seed=22)
    out = []
    for z in (None, a[:, :, None].expand(T, H, D).reshape(T, H * D).contiguous()):
        st = rnd(3, H, Dv, D, seed=23, scale=0.3)
        o = torch.zeros(T, H, Dv, device=DEV)
        ops.delta_scan(q, k, v, b, a if z is None else None, a_log, dt_bias if z is None else dt_bias[:, None].expand(H, D).reshape(-1).contiguous(),
                       D ** -0.5, 1e-6, st, slots, info, 2, o, z=z)
        out.append((o, st))
    for x, y in zip(*out):
        torch.testing.assert_close(x, y, rtol=1e-4, atol=1e-5)


@pytest.mark.parametrize("cuts", [[700], [333, 2, 365], [64, 64, 1, 1, 570], [699, 1], [16, 17, 15, 1, 651], [1] * 10 + [690]])
def test_one_channel_keeps_a_value_for_hundreds_of_tokens_and_its_neighbour_forgets_it(cuts):
    """Tokens 3 and 4 write values along channels 0 and 1, which no later token touches.  Channel 0 hardly decays, channel 1
    loses half per token; tokens 698 and 699 ask for them.  A state lost or restarted at any cut, or a decay of the wrong
    channel, shows."""
    H, G, D, Dv, T = 2, 1, 16, 8, 700
    g = torch.Generator().manual_seed(5)
    k = torch.zeros(T, D)
    k[:, 2:] = torch.randn(T, D - 2, generator=g)
    q = torch.randn(T, D, generator=g) * 0.1
    for t, c in ((3, 0), (4, 1)):
        k[t] = 0
        k[t, c] = 5.0
    for t, c in ((5, 1), (698, 1), (699, 0)):
        q[t] = 0
        q[t, c] = 4.0
    v = torch.randn(T, H * Dv, generator=g)
    v[3] = torch.arange(1, H * Dv + 1).float()
    v[4] = -torch.arange(1, H * Dv + 1).float()
    b = torch.full((T, H), 4.0)            # beta near one
    z = torch.full((T, H * D), -9.0)       # softplus near zero: decays near one
    z.view(T, H, D)[:, :, 1] = 0.0         # softplus(0) = ln 2: a half
    a_log, dt_bias = torch.zeros(H), torch.zeros(H * D)
    dev = lambda t: t.to(DEV).contiguous()  # noqa: E731
    state = torch.full((2, H, Dv, D), 3.0, device=DEV)
    outs, i = [], 0
    for c in cuts:
        info, slots, _ = segs([(c, i + c)])
        o = torch.zeros(c, H, Dv, device=DEV)
        ops.delta_scan(dev(q[i:i + c]), dev(k[i:i + c]), dev(v[i:i + c]), dev(b[i:i + c]), None, dev(a_log), dev(dt_bias), 1.0, 1e-6, state,
                       slots, info, 1, o, z=dev(z[i:i + c]))
        outs.append(o)
        i += c
    assert i == T
    got = torch.cat(outs).cpu().reshape(T, -1)
    beta = float(torch.sigmoid(torch.tensor(4.0)))
    kept = beta * float(torch.exp(-torch.nn.functional.softplus(torch.tensor(-9.0)))) ** (T - 4)
    torch.testing.assert_close(got[699], v[3] * kept, rtol=1e-2, atol=0.05)
    torch.testing.assert_close(got[5], v[4] * beta * 0.5, rtol=1e-2, atol=0.05)
    assert float(got[698].abs().max()) < 1e-6


def test_delta_scan_takes_one_kind_of_decay():
    q, k, v, b, z, a_log, dt_bias = delta_case(torch.float32, 2, 1, 8, 8, 3)
    info, slots, _ = segs([(3, 3)])
    st, o = torch.zeros(2, 2, 8, 8, device=DEV), torch.zeros(3, 2, 8, device=DEV)
    for a, zz in ((None, None), (b, z)):
        with pytest.raises(KernelError):
            ops.delta_scan(q, k, v, b, a, a_log, dt_bias, 1.0, 1e-6, st, slots, info, 1, o, z=zz)


# --------------------------------------------------------------------------- retention
def retention_case(dtype, H, D, Dv, n_rot, lens, seed=0, max_pos=None):
    info, slots, T = segs(lens)
    rows = rnd(T, 2 * H * D + H * Dv + 5, dtype=dtype, seed=seed, scale=0.5)
    longest = max_pos or max(kv for _, kv in lens)
    ang = torch.arange(longest)[:, None] * 0.61 ** torch.arange(max(n_rot // 2, 1))[None, :]
    table = torch.cat([ang.cos(), ang.sin()], -1).float().to(DEV) if n_rot else None
    decay = (1.0 - torch.logspace(-3.5, -0.5, H)).to(DEV)
    return rows[:, :H * D], rows[:, H * D:2 * H * D], rows[:, 2 * H * D:2 * H * D + H * Dv], decay, table, info, slots, T


def run_retention(q, k, v, decay, table, info, slots, lens, state, chunk, neighbours, T, H, D, Dv):
    chunks, per_seg, single, multi = chunk_list(lens, chunk)
    n = chunks.shape[0]
    carry = torch.full((n, H, D, Dv), float("nan"), device=DEV) if multi else None
    prod = torch.full((n, H, D), float("nan"), device=DEV) if multi else None
    out = torch.full((T, H, Dv), float("nan"), device=DEV)
    ops.gla_scan(q, k, v, None, None, 1.0, D ** -0.5, state, slots, info, len(lens), torch.from_numpy(chunks).to(DEV), n,
                 torch.from_numpy(per_seg).to(DEV), single, multi, carry, prod, out, a_head=decay, rope_table=table, neighbours=neighbours)
    return out


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,Dv,n_rot", [(2, 16, 24, 16), (4, 48, 64, 32), (1, 130, 33, 130), (3, 10, 14, 6), (2, 128, 128, 128),
                                          (1, 256, 40, 64), (5, 8, 8, 4), (2, 64, 32, 0), (3, 64, 64, 60)])
@pytest.mark.parametrize("neighbours", [False, True])
def test_retention_against_the_stated_recurrence(dtype, H, D, Dv, n_rot, neighbours):
    """One row of decays for every token; rotation inside the kernel, in every way it reads the rows: bfloat16 rows fetched
    ahead, few rows straight from memory, sizes that allow no wide reads, 32-bit rows."""
    lens = [(1, 9), (130, 130), (64, 200), (65, 65), (2, 2), (1, 1), (15, 300)]
    q, k, v, decay, table, info, slots, T = retention_case(dtype, H, D, Dv, n_rot, lens)
    state = rnd(len(lens) + 1, H, D, Dv, seed=7)
    want, st_want = torch.zeros(T, H, Dv), state.cpu().clone()
    ref.gla_scan(q.cpu(), k.cpu(), v.cpu(), None, None, 1.0, D ** -0.5, st_want, slots.cpu(), info.cpu(), len(lens), None, 0, None, True,
                 True, None, None, want, a_head=decay.cpu(), rope_table=None if table is None else table.cpu(), neighbours=neighbours)
    for chunk in (64, 16, 300):
        st = state.clone()
        got = run_retention(q, k, v, decay, table, info, slots, lens, st, chunk, neighbours, T, H, D, Dv)
        torch.testing.assert_close(got.cpu(), want, rtol=2e-4, atol=2e-4)
        torch.testing.assert_close(st.cpu(), st_want, rtol=2e-4, atol=2e-4)


@pytest.mark.parametrize("cuts", [[900], [64, 2, 65, 63, 706], [1] * 20 + [880], [899, 1], [450, 450]])
def test_retention_reads_a_token_by_its_distance_alone(cuts):
    """Every query and key is the same row: o_t = sum_s a^(t-s) (q' R_(t-s) k') v_s, whatever the positions' cut; with one value
    that stands out (token 7) and a head that hardly decays, token 899 still reads it."""
    H, D, Dv, T, n_rot = 2, 16, 8, 900, 16
    decay = torch.tensor([0.999, 0.8], device=DEV)
    row_q, row_k = rnd(H, D, seed=3), rnd(H, D, seed=4)
    v = rnd(T, H * Dv, seed=5, scale=0.01)
    v[7] = 100.0
    ang = torch.arange(T).double()[:, None] * 0.61 ** torch.arange(n_rot // 2).double()[None, :]
    table = torch.cat([ang.cos(), ang.sin()], -1).float().to(DEV)
    state, outs, i = torch.full((2, H, D, Dv), 5.0, device=DEV), [], 0
    for c in cuts:
        info, slots, _ = segs([(c, i + c)])
        outs.append(run_retention(row_q.expand(c, H, D).reshape(c, -1).contiguous(), row_k.expand(c, H, D).reshape(c, -1).contiguous(),
                                  v[i:i + c], decay, table, info, slots, [(c, i + c)], state, 64, False, c, H, D, Dv))
        i += c
    assert i == T
    got = torch.cat(outs).double().cpu()
    half = n_rot // 2
    a, b = row_q.double().cpu(), row_k.double().cpu()
    x = (a[:, :half] * b[:, :half] + a[:, half:] * b[:, half:])
    y = (a[:, :half] * b[:, half:] - a[:, half:] * b[:, :half])
    dots = (ang.cos() @ x.T + ang.sin() @ y.T) * D ** -0.5           # [distance, head]
    for t in (7, 8, 100, 512, 899):
        w = dots[: t + 1] * decay.double().cpu()[None, :] ** torch.arange(t + 1).double()[:, None]
        want = torch.einsum("dh,dhv->hv", w.flip(0), v.double().cpu().view(T, H, Dv)[: t + 1])
        torch.testing.assert_close(got[t], want, rtol=1e-3, atol=1e-3)


# --------------------------------------------------------------------------- experts in groups
@pytest.mark.parametrize("T,E,k,count,keep,extra", [(1, 8, 2, 4, 2, 1), (7, 6, 2, 3, 1, 0), (32, 64, 8, 8, 3, 1), (5, 16, 4, 2, 1, 1),
                                                    (40, 250, 6, 10, 4, 1), (33, 512, 8, 64, 5, 0), (3, 640, 5, 32, 2, 1), (9, 12, 3, 12, 5, 1),
                                                    (6, 96, 4, 3, 3, 0)])
@pytest.mark.parametrize("scoring", ["softmax_raw", "softmax", "sigmoid"])
def test_routing_within_the_best_groups(T, E, k, count, keep, extra, scoring):
    H = 64
    x = rnd(T, H, seed=1)
    w = rnd(E + extra, H, seed=2, scale=H ** -0.5 * 2)
    bias = rnd(E, seed=3, scale=0.05) if scoring == "sigmoid" else None
    logits = x.cpu() @ w.cpu().T
    mk = lambda d: (torch.zeros(T, k, dtype=torch.int32, device=d), torch.zeros(T, k, device=d), torch.zeros(T, 2, device=d))  # noqa: E731
    ids, wts, aux = mk("cpu")
    ref.router_topk(logits, cpu(bias), k, scoring, 1.0, ids, wts, n_extra=extra, aux=aux, groups=(count, keep))
    if keep < count:  # (the groups matter: without them the choice is another one somewhere)
        size = E // count
        assert all(len({int(e) // size for e in row}) <= keep for row in ids)
        free = torch.zeros_like(ids)
        ref.router_topk(logits, cpu(bias), k, scoring, 1.0, free, torch.zeros(T, k), n_extra=extra, aux=torch.zeros(T, 2))
        assert T < 5 or size == 1 or not torch.equal(free, ids)
    i2, w2, a2 = mk(DEV)
    parts = torch.cat([torch.nn.functional.pad(logits * f, (0, 3), value=1e9) for f in (0.75, 0.25)], -1).to(DEV).contiguous()
    for lg, n_parts, pad in ((logits.to(DEV), 1, 0), (parts, 2, 3)):
        ops.router_topk(lg, bias, k, scoring, 1.0, i2, w2, n_parts=n_parts, n_extra=extra, aux=a2, n_pad=pad, groups=(count, keep))
        torch.testing.assert_close(i2.cpu(), ids, rtol=0, atol=0)
        torch.testing.assert_close(w2.cpu(), wts, rtol=1e-5, atol=1e-6)
        torch.testing.assert_close(a2.cpu(), aux, rtol=1e-5, atol=1e-6)
    if not ops.moe_route_fits(T, H, E, k):
        return
    i2, w2, a2 = mk(DEV)
    ops.moe_route(x, w, bias, k, scoring, 1.0, torch.zeros(T, E + extra, device=DEV), i2, w2, n_extra=extra, aux=a2, groups=(count, keep))
    torch.testing.assert_close(i2.cpu(), ids, rtol=0, atol=0)
    torch.testing.assert_close(w2.cpu(), wts, rtol=1e-4, atol=1e-5)


def test_routing_refuses_groups_that_do_not_fit():
    lg, ids, wts = rnd(3, 12), torch.zeros(3, 4, dtype=torch.int32, device=DEV), torch.zeros(3, 4, device=DEV)
    for groups in ((5, 2), (4, 5), (4, 1), (0, 0)):
        with pytest.raises(KernelError):
            ops.router_topk(lg, None, 4, "softmax_raw", 1.0, ids, wts, groups=groups)


# --------------------------------------------------------------------------- two scaled results, experts with a gated shared row
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,C", [(5, 64), (9, 90), (3, 21), (4, 1030), (6, 3072), (70, 2048), (2, 12288)])
def test_results_join_the_stream_without_a_norm_of_their_own(dtype, T, C):
    k = 3
    y, y2, shared = (rnd(T, C, dtype=dtype, seed=i) for i in (1, 2, 3))
    rows = rnd(T * k, C, dtype=dtype, seed=5)
    pos = torch.randperm(T * k, generator=torch.Generator().manual_seed(6)).to(torch.int32).view(T, k).to(DEV)
    aux = torch.rand(T, 2, generator=torch.Generator().manual_seed(7)).to(DEV)
    wr = rnd(C, seed=11) * 0.3 + 1.0
    picked = torch.tensor([T - 1, 0], dtype=torch.int32, device=DEV)
    for kw in (dict(x=y, x2=y2, scales=(0.7, -1.3)), dict(x=y), dict(x=rows, routed=(pos, k, shared, aux, None)),
               dict(x=rows, routed=(pos, k, None, None, None)), dict(x=y, x2=y2, scales=(0.5, 2.0), rows=picked),
               dict(x=rows, routed=(pos, k, shared, aux, None), rows=picked)):
        n = 2 if "rows" in kw else T
        for normed in (True, False):
            if not normed and "rows" in kw:
                continue
            res = [rnd(T, C, seed=12), rnd(T, C, seed=12).cpu()]
            out = [torch.zeros(n, C, dtype=dtype, device=d) for d in (DEV, "cpu")]
            f32 = [torch.zeros(n, C, device=d) for d in (DEV, "cpu")]
            for i, fn in enumerate((ops.stream_step, ref.stream_step)):
                mv = (lambda t: t) if i == 0 else cpu
                args = {a: mv(b) for a, b in kw.items()}
                if normed:
                    args.update(pre_weight=mv(wr), pre_eps=1e-6, out=out[i], norm_f32=f32[i], f32_rounded=True)
                fn(res[i], **args)
            torch.testing.assert_close(res[0].cpu(), res[1], rtol=1e-6, atol=2e-6, msg=lambda m: f"{sorted(kw)}: stream: {m}")
            torch.testing.assert_close(out[0].float().cpu(), out[1].float(), **tol(dtype))
            torch.testing.assert_close(f32[0], out[0].float(), rtol=0, atol=0)  # the 32-bit copy is the rounded row


# --------------------------------------------------------------------------- the engine against the plain model
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G1", "G2", "G3", "G4", "G5"])
def test_cuts_and_batches_agree_with_the_plain_model(name, dtype, tmp_path_factory):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainGizulorn(folder)
    eng = make_engine(folder, dtype, DEV, 16 if name == "G3" else PAGE, pages=40)
    toks = tokens_for(plain.vocab, 70, 11)
    want = plain.logits(toks)
    check_rows(replay_whole(eng, "w", toks), plain, toks, dtype, "whole", want=want)
    check_rows(replay_cuts(eng, "d", toks, [38]), plain, toks, dtype, "last 32 one by one", want=want)
    check_rows(replay_cuts(eng, "c", toks, [7, 2, 13, 2, 5, 3, 2, 11, 2]), plain, toks, dtype, "portions", want=want)
    check_rows(replay_cuts(eng, "one", toks[:40], []), plain, toks, dtype, "one by one from the first token", want=want)
    eng.cache.check()
    eng.check_kernels()
    assert all(g.pool.free_count == g.pool.num_pages for g in eng.cache.paged)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G1", "G4"])
def test_mixed_steps_with_few_pages_and_slots(name, dtype, tmp_path_factory):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainGizulorn(folder)
    lengths = {"r0": 45, "r1": 60, "r2": 38, "r3": 52, "r4": 41, "r5": 47}
    seqs = {r: tokens_for(plain.vocab, n, i) for i, (r, n) in enumerate(lengths.items())}
    eng = make_engine(folder, dtype, DEV, PAGE, pages=4 * (-(-64 // PAGE)), max_step=40)
    got = replay_mixed(eng, seqs, mixed_schedule(lengths, seed=3))
    for r, toks in seqs.items():
        check_rows(got[r], plain, toks, dtype, r)
    assert any(g.pool.handed_out > g.pool.num_pages for g in eng.cache.paged), "the trace was meant to use pages again"
    assert eng.cache.slots.free_count == 4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["G1", "G3", "G4"])
def test_long_prompt_long_decoding_and_recorded_steps(name, dtype, tmp_path_factory):
    """Hundreds of tokens across many pages and windows, a hundred tokens one by one (recorded into a CUDA graph at the
    first), and a long step in between."""
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainGizulorn(folder)
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
    folder = model_folder(tmp_path_factory.getbasetemp(), "G3", GIZU_3)
    plain = PlainGizulorn(folder)
    toks = tokens_for(plain.vocab, 420, 9)
    want = plain.logits(toks)
    eng = make_engine(folder, "bfloat16", DEV, 16, pages=96, max_step=512)
    ops.variant_counts(reset=True)
    check_rows(replay_whole(eng, "w", toks), plain, toks, "bfloat16", "whole", want=want)
    forms = ops.variant_counts()
    assert forms.get("attention: tcgen05, 128-row query tiles, window or sink", 0) == 1, forms
    ops.variant_counts(reset=True)
    check_rows(replay_cuts(eng, "c", toks, [250, 130, 2]), plain, toks, "bfloat16", "portions, the rest one by one", want=want)
    assert eng.graphs and not any("mma.sync, 16-row" in k for k in ops.variant_counts())  # single tokens too
    others = {f"o{i}": tokens_for(plain.vocab, 20 + i, 20 + i) for i in range(3)}
    for r, t in others.items():  # three requests that decode beside a long portion
        eng.step([StepEntry(r, t[:-1], [])])
    out = eng.step([StepEntry("long", toks[:200], list(range(200)))] + [StepEntry(r, t[-1:], [0]) for r, t in others.items()])
    check_rows(out.logits[:200].float().cpu(), plain, toks, "bfloat16", "a long portion beside single tokens", want=want)
    for i, (r, t) in enumerate(others.items()):
        assert float(row_error(out.logits[200 + i:201 + i].float().cpu(), plain.logits(t)[-1:]).max()) < 1.5, r
    eng.check_kernels()


REAL_LAYERS = {  # layers of the size of a real model's (no test of the tiny configurations reaches these kernel forms)
    "architecture": "Gizulorn", "vocab": 8192, "width": 2048, "norm": {"eps": 1e-6},
    "layers": [
        {"type": "parallel", "mixer": {
            "left": {"heads": 16, "kv_heads": 4, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "mask": {"size": 256, "keep_first": 4},
                     "rot": {"dims": 128, "base": 500000.0, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}},
            "right": {"heads": 16, "kv_heads": 8, "dim": 128, "vdim": 128, "conv": 4, "decay_rank": 64, "gate_rank": 128},
            "left_scale": 0.9, "right_scale": 1.1},
         "mlp": {"kind": "dense", "ff": 4096}},
        {"type": "retention", "mixer": {"heads": 8, "dim": 128, "vdim": 256, "decay": [1.0 - 2.0 ** -(5 + i) for i in range(8)],
                                        "rot": {"dims": 128, "base": 10000.0}},
         "mlp": {"kind": "moe", "expert": {"ff": 768}, "router": {"experts": 32, "top": 4, "groups": {"count": 4, "keep": 2}},
                 "shared": {"ff": 1024}}},
    ]}


def test_layers_of_real_sizes_agree_across_cuts_and_dtypes():
    """Heads of 128, long portions: the attention kernel's tcgen05 form, expert products on the tensor cores, the delta rule in
    its form for many columns.  No plain model at these sizes: the 32-bit engine is compared with itself across cuts, the
    bfloat16 engine with it."""
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
            assert forms.get("attention: tcgen05, 128-row query tiles, window or sink", 0) == 1, forms
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

    folder = model_folder(tmp_path_factory.getbasetemp(), "G1", GIZU_1)
    plain = PlainGizulorn(folder)
    prompts = [[5, 17, 3, 150, 41], [9, 8, 7, 6, 5, 4, 3, 2, 1, 0, 11, 12], [199]]
    for dtype in ("float32", "bfloat16"):
        llm = LLM(folder, dtype=dtype, device=DEV, page_size=4, num_page_override=48, max_step_tokens=8,
                  max_extend_tokens=8, max_running_req=2)  # three prompts on two request slots, in portions of eight
        outs = llm.generate(prompts, SamplingParams(max_tokens=20))
        for p, o in zip(prompts, outs):
            toks = list(p)
            assert len(o["token_ids"]) == 20
            for got in o["token_ids"]:
                logits = plain.logits(toks)[-1]
                top2 = torch.topk(logits, 2).values
                if dtype == "float32" or float(top2[0] - top2[1]) > 0.3:
                    assert got == int(torch.argmax(logits)), (dtype, p, o)
                toks.append(got)


def test_the_replay_tool_runs_the_design(tmp_path_factory, tmp_path):
    folder = model_folder(tmp_path_factory.getbasetemp(), "G4", ALL["G4"])
    plain = PlainGizulorn(folder)
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
