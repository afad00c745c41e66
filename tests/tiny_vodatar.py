"""Tiny Vodatar configurations for tests; they differ in every size, option and constant.

V1: the middle two of four layers run twice; both mixers, values wider than two maps, two norm groups, taps of 3 (projections)
    and 4 (inputs), identity experts and a shared expert, a layer without feed-forward inside the loop.
V2: nothing is a multiple of 4: width 90 in three norm groups, vocabulary 101, one head, a map of 10 of which 6 dimensions
    turn, values narrower than a map; one tap everywhere (no convolution state at all); the loop is the whole stack, once;
    no soft cap, no identity experts, a factor of 1; plain rotation frequencies in the latent layer.
V3: the whole stack of two layers three times over; a cached latent row of 128 and two maps of 64 on values of 128 (the
    tensor-core attention kernels' size); sharp attention (large score scales), so that a key one place off moves the
    logits; one norm group; two taps; one expert a token, of which one in five hands the input back.
V4: no loop; five taps; twelve norm groups; six heads on three key heads; more identity experts than a token's choices leave
    out; a soft cap that most scores feel; no shared expert in one layer; a strong stretch of the rotation frequencies.
"""

from __future__ import annotations

ARCH = "Vodatar"
PAGE = 4


def _att(heads, kv_heads, dim, vdim, conv, scale, softcap, diff, rot_dims, base):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "scale": scale, "diff": diff,
         "rot": {"dims": rot_dims, "base": base}}
    if softcap is not None:
        m["softcap"] = softcap
    return "attention", m


def _latent(heads, dim, rot_dim, vdim, kv_rank, scale, base, scaling=None):
    rot = {"dims": rot_dim, "base": base}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                "scale": scale, "rot": rot}


def _moe(ff, experts, identity, top, shared):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top}}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def _model(vocab, width, eps, groups, mult, taps, loop, layers):
    raw = {"architecture": ARCH, "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
           "residual_mult": mult, "canon": {"taps": taps},
           "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop is not None:
        raw["loop"] = dict(zip(("start", "stop", "times"), loop))
    return raw


VODA_1 = _model(200, 64, 1e-5, 2, 0.6, 4, (1, 3, 2), [
    (_att(4, 2, 8, 20, 3, 0.4, 9.0, 0.2, 8, 1000.0), _moe(40, 6, 2, 2, 48)),
    (_latent(3, 8, 8, 12, 20, 0.3, 100.0, (2.0, 64, 8.0, 1.0)), None),
    (_att(2, 2, 16, 24, 3, 0.25, 12.0, 0.4, 12, 500.0), _moe(24, 5, 1, 3, 32)),
    (_latent(2, 12, 4, 20, 16, 0.25, 50.0, (3.0, 128, 4.0, 0.5)), _moe(32, 4, 2, 2, 40)),
])

VODA_2 = _model(101, 90, 1e-6, 3, 1.0, 1, (0, 3, 1), [
    (_latent(1, 14, 6, 18, 22, 0.3, 300.0), _moe(26, 3, 0, 2, 30)),
    (_att(1, 1, 10, 7, 1, 0.35, None, 0.1, 6, 70.0), _moe(30, 4, 0, 3, 22)),
    (_att(1, 1, 10, 22, 1, 0.3, 5.0, 0.6, 10, 70.0), None),
])

VODA_3 = _model(160, 96, 1e-5, 1, 0.4, 2, (0, 2, 3), [
    (_latent(6, 16, 32, 16, 96, 0.7, 10000.0, (4.0, 256, 32.0, 1.0)), _moe(64, 4, 1, 1, 80)),
    (_att(3, 1, 64, 128, 4, 0.5, 30.0, 0.3, 64, 5000.0), _moe(48, 4, 1, 1, 64)),
])

VODA_4 = _model(120, 72, 1e-5, 12, 0.5, 5, None, [
    (_att(6, 3, 12, 28, 5, 0.5, 2.0, 0.5, 8, 200.0), _moe(36, 3, 3, 4, None)),
    (_latent(4, 8, 16, 10, 30, 0.25, 400.0, (16.0, 32, 2.0, 0.25)), _moe(24, 7, 5, 3, 28)),
    (_att(4, 1, 6, 12, 2, 0.6, 3.0, 0.25, 6, 30.0), _moe(28, 3, 1, 2, 36)),
])

ALL = {"V1": VODA_1, "V2": VODA_2, "V3": VODA_3, "V4": VODA_4}
