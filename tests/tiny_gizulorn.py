"""Tiny Gizulorn configurations for tests; they differ in every size, option and constant.

G1: both mixers; a window of 9 that keeps 3 tokens (less than a page), values wider than keys, part of each head rotated with
    scaled frequencies; delta heads in pairs on a key head, three taps; experts in three groups of which two are open; a
    layer without feed-forward.
G2: nothing is a multiple of 4: width 90, vocabulary 101, one query head, low ranks of 5 and 7, one tap (no convolution
    state), a window of one token that keeps one; values narrower than keys; retention with three heads; one group, one
    expert a token, no shared expert.
G3: heads of 128 in every mixer (the tensor-core attention kernels' size), six query heads on two key heads, a window of 130
    that keeps 6, delta heads on keys of their own; sharp attention, so that a key one place off moves the logits; top 3
    of 8 experts in four groups.
G4: a window of 6 that keeps 21 tokens (more than the window, more than a page, more than one quantum of the 32-bit
    kernel's pages), no rotation in the attention, five taps, more query heads than a tile has rows on one key head; decays of 1 and of
    almost nothing; layers of dense feed-forwards only.
G5: no window at all, interleaved rotation of everything; every group open.
"""

from __future__ import annotations

ARCH = "Gizulorn"
PAGE = 4


def _rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return r


def _pair(left, right, scales):
    heads, kv, dim, vdim, mask, rot, scale = left
    le = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if mask is not None:
        le["mask"] = {"size": mask[0], "keep_first": mask[1]}
    if rot is not None:
        le["rot"] = rot
    heads, kv, dim, vdim, conv, ranks = right
    ri = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "decay_rank": ranks[0], "gate_rank": ranks[1]}
    return "parallel", {"left": le, "right": ri, "left_scale": scales[0], "right_scale": scales[1]}


def _ret(heads, dim, vdim, decay, rot):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}
    if rot is not None:
        m["rot"] = rot
    return "retention", m


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(ff, experts, top, groups, shared):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups is not None:
        m["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, eps, layers):
    return {"architecture": ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps},
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


GIZU_1 = _model(200, 64, 1e-5, [
    (_pair((4, 2, 16, 24, (9, 3), _rot(8, 1000.0, (2.0, 1.0, 4.0, 64)), 0.4), (4, 2, 12, 20, 3, (10, 6)), (0.7, 1.2)),
     _moe(40, 6, 2, (3, 2), 48)),
    (_ret(2, 16, 20, [0.96, 0.999], _rot(12, 500.0)), None),
    (_ret(3, 8, 12, [0.9, 0.99, 0.9995], _rot(8, 100.0)), _moe(24, 8, 3, (2, 1), 32)),
    (_pair((2, 1, 20, 12, (17, 1), _rot(20, 200.0, (8.0, 0.5, 2.0, 32)), 0.3), (2, 2, 16, 8, 2, (4, 12)), (1.3, 0.6)), _dense(72)),
])

GIZU_2 = _model(101, 90, 1e-6, [
    (_ret(3, 10, 14, [0.97, 0.5, 0.998], _rot(6, 70.0)), _moe(26, 3, 1, None, None)),
    (_pair((1, 1, 14, 10, (1, 1), _rot(6, 300.0, (3.0, 1.0, 2.0, 100)), 0.35), (3, 1, 10, 6, 1, (5, 7)), (1.0, -0.5)), _dense(30)),
    (_ret(1, 6, 18, [0.995], None), None),
])

GIZU_3 = _model(160, 96, 1e-5, [
    (_pair((6, 2, 128, 128, (130, 6), _rot(128, 10000.0, (4.0, 1.0, 4.0, 256)), 0.3), (2, 2, 128, 64, 4, (16, 8)), (0.5, 0.9)),
     _moe(64, 8, 3, (4, 2), 80)),
    (_ret(2, 128, 64, [0.98, 0.9999], _rot(128, 5000.0)), _moe(48, 4, 2, (4, 3), 64)),
])

GIZU_4 = _model(120, 72, 1e-5, [
    (_pair((20, 1, 8, 8, (6, 21), None, 0.6), (6, 3, 24, 12, 5, (3, 9)), (0.9, 1.0)), _dense(60)),
    (_ret(2, 12, 28, [1.0, 0.01], _rot(4, 30.0)), _dense(40)),
    (_pair((3, 3, 12, 28, (33, 70), _rot(8, 400.0), 0.5), (1, 1, 40, 36, 4, (8, 8)), (0.4, 1.5)), None),
])

GIZU_5 = _model(96, 48, 1e-5, [
    (_pair((4, 4, 32, 32, None, _rot(32, 2000.0), 0.25), (4, 1, 32, 16, 4, (6, 5)), (1.1, 0.8)), _moe(28, 4, 2, (2, 2), 20)),
])

ALL = {"G1": GIZU_1, "G2": GIZU_2, "G3": GIZU_3, "G4": GIZU_4, "G5": GIZU_5}
