"""Gizulorn without a GPU: its config reader, model description and checkpoint names, what the cache keeps of a window with
kept first tokens, the plain statements of its mechanisms against other ways of writing them, and the engine's step, cache,
state and batching logic with the plain PyTorch statements of the kernels (tests/kernel_refs.py) standing in for the CUDA
kernels."""

import copy
import math

import numpy as np
import pytest
import torch

import kernel_refs
from helpers import make_engine, mixed_schedule, model_folder, replay_cuts, replay_mixed, replay_whole, tokens_for
from plain import gizulorn_plain as plain_model
from plain.gizulorn_plain import PlainGizulorn
from tiny_gizulorn import ALL, GIZU_1, GIZU_2, GIZU_3, GIZU_4, GIZU_5, PAGE

from freetoken_b200.cache.manager import CacheManager
from freetoken_b200.config.spec import PagedKVNeed, PartSpec, StateNeed
from freetoken_b200.engine.attention_plan import SPLIT_QUANTUM, build_plan
from freetoken_b200.engine.build import describe_model
from freetoken_b200.engine.engine import StepEntry
from freetoken_b200.errors import ConfigError
from freetoken_b200.registry import architecture_of

TOL = dict(rtol=1e-4, atol=5e-5)


@pytest.fixture
def cpu_ops(monkeypatch):
    kernel_refs.install(monkeypatch)


def build_model(raw):
    from freetoken_b200.models.model import Model
    from freetoken_b200.parts import BuildEnv, Workspace

    _, _, spec, _ = describe_model(raw)
    cpu = torch.device("cpu")
    return Model(spec, BuildEnv(dtype=torch.float32, device=cpu, max_seq_len=64, max_step_tokens=8, workspace=Workspace(cpu)))


# --------------------------------------------------------------------------- config, description, names
def test_the_description_follows_the_config():
    _, cfg, spec, expected = describe_model(GIZU_1)
    assert [l.mixer.kind for l in spec.layers] == ["side_by_side", "retention", "retention", "side_by_side"]
    assert [l.ffn.kind for l in spec.layers] == ["moe", "none", "moe", "gated_mlp"]
    assert all(l.block.kind == "prenorm_residual" for l in spec.layers)
    m = spec.layers[0].mixer
    assert m["scales"] == (0.7, 1.2)
    (ln, le), (rn, ri) = m["branches"]
    assert (ln, rn) == ("left", "right") and (le.kind, ri.kind) == ("gqa_attention", "gated_delta")
    assert (le["window"], le["keep_first"], le["scale"], le["sink"], le["v_head_dim"]) == (9, 3, 0.4, "learned", 24)
    assert le["position"].kind == "rope_interleaved" and le["position"]["band_scaling"] == (2.0, 1.0, 4.0, 64.0)
    assert (ri["n_kv_heads"], ri["taps"], ri["decay_rank"], ri["gate_rank"], ri["gate"]) == (2, 3, 10, 6, "sigmoid")
    r = spec.layers[2].mixer
    assert r["decay"] == (0.9, 0.99, 0.9995) and r["position"].kind == "rope_neox" and r["position"]["rotary_dim"] == 8
    f = spec.layers[2].ffn
    assert (f["n_experts"], f["top_k"], f["groups"], f["scoring"], f["shared_inter"], f["shared_gate"]) == (8, 3, (2, 1), "softmax_raw", 32, True)
    assert expected["l0.mix.left.qkv_proj.weight"].shape == (4 * 16 + 2 * 16 + 2 * 24, 64)
    assert expected["l0.mix.left.sink"].shape == (4,)
    assert expected["l0.mix.right.in_proj.weight"].shape == (2 * 2 * 12 + 4 * 20 + 6 + 4 + 10, 64)
    assert expected["l0.mix.right.conv.weight"].shape == (2 * 2 * 12 + 4 * 20, 3)
    assert expected["l0.mix.right.decay_proj.weight"].shape == (48, 10) and expected["l0.mix.right.gate_proj.weight"].shape == (80, 6)
    assert expected["l0.mix.right.dt_bias"].shape == (48,) and expected["l0.mix.right.A_log"].shape == (4,)
    assert "l1.norm2.weight" not in expected and "l0.norm2.weight" in expected
    assert expected["l1.mix.in_proj.weight"].shape == (2 * 2 * 16 + 2 * 2 * 20, 64)
    assert expected["l0.mlp.shared_gate.weight"].shape == (1, 64) and expected["l3.mlp.gate_up_proj.weight"].shape == (144, 64)
    _, _, spec2, expected2 = describe_model(GIZU_2)
    assert spec2.layers[0].ffn["groups"] == (1, 1) and "l0.mlp.shared_gate.weight" not in expected2
    assert spec2.layers[2].mixer["position"].kind == "none"
    left = describe_model(GIZU_5)[2].layers[0].mixer["branches"][0][1]
    assert left["window"] is None and left["keep_first"] == 0


def test_the_checkpoint_names_are_the_designs(tmp_path_factory):
    from freetoken_b200.weights.safetensors_io import ModelFolder

    mf = ModelFolder(model_folder(tmp_path_factory.getbasetemp(), "G1", GIZU_1))
    names = set(mf.names())
    right = [f"l0.mix.right.{n}" for n in ("q", "q.conv", "k", "k.conv", "v", "v.conv", "b", "A_log", "norm", "a1", "a2", "dt_bias",
                                          "g1", "g2", "o")]
    left = [f"l0.mix.left.{n}" for n in ("q", "k", "v", "sink", "o")]
    assert {n for n in names if n.startswith("l0.mix.")} == set(left + right)
    assert {n for n in names if n.startswith("l1.")} == {"l1.norm1"} | {f"l1.mix.{n}" for n in "qkvgo"}
    assert {n for n in names if n.startswith("l3.mlp")} == {"l3.mlp.gate", "l3.mlp.up", "l3.mlp.down"}
    for n in ("embed", "head", "final.norm", "l0.norm1", "l0.norm2", "l0.mlp.e5.down", "l0.mlp.router", "l0.mlp.shared.sg",
              "l0.mlp.shared.up"):
        assert n in names, n
    assert {mf.dtype(n) for n in names} == {torch.bfloat16}


def test_the_low_ranks_come_from_the_weight_file(tmp_path_factory):
    from freetoken_b200.engine.build import typed_config

    folder = model_folder(tmp_path_factory.getbasetemp(), "G2", GIZU_2)
    raw = copy.deepcopy(GIZU_2)
    for k in ("decay_rank", "gate_rank"):
        del raw["layers"][1]["mixer"]["right"][k]
    arch = architecture_of(raw)
    assert arch.parse_config(raw).layers[1].mixer.right.decay_rank == 0
    right = typed_config(arch, raw, folder).layers[1].mixer.right
    assert (right.decay_rank, right.gate_rank) == (5, 7)


def test_config_errors_name_the_key():
    def broken(path, value, delete=False):
        raw = copy.deepcopy(GIZU_1)
        d = raw
        for k in path[:-1]:
            d = d[k]
        if delete:
            del d[path[-1]]
        else:
            d[path[-1]] = value
        return raw

    left, right = ["layers", 0, "mixer", "left"], ["layers", 0, "mixer", "right"]
    for raw, word in [
        (broken(["vocab"], None, True), "vocab"),
        (broken(["norm", "eps"], None, True), "eps"),
        (broken(["layers", 0, "type"], "conv"), "type"),
        (broken(["layers", 0, "mixer", "left_scale"], None, True), "left_scale"),
        (broken(left + ["kv_heads"], 3), "kv_heads"),
        (broken(left + ["mask", "size"], 0), "mask.size"),
        (broken(left + ["mask", "keep_first"], -1), "keep_first"),
        (broken(left + ["rot", "dims"], 18), "rot.dims"),
        (broken(left + ["rot", "scaling", "high"], None, True), "scaling.high"),
        (broken(right + ["conv"], 0), "conv"),
        (broken(right + ["heads"], 3), "heads"),
        (broken(["layers", 1, "mixer", "decay"], [0.5]), "decay"),
        (broken(["layers", 1, "mixer", "decay"], None, True), "decay"),
        (broken(["layers", 0, "mlp", "router", "top"], 5), "router.top"),
        (broken(["layers", 0, "mlp", "router", "groups", "keep"], 4), "groups"),
        (broken(["layers", 0, "mlp", "router", "groups", "count"], 4), "groups"),
        (broken(["layers", 3, "mlp", "kind"], "glu"), "kind"),
    ]:
        with pytest.raises(ConfigError, match=word):
            architecture_of(raw).parse_config(raw)


def test_pages_and_states():
    model = build_model(GIZU_1)
    needs = dict(model.cache_needs())
    assert needs[(0, 0)] == PagedKVNeed((("k", 2, 32), ("v", 2, 32)), 9, 3)
    assert needs[(0, 1)] == StateNeed((("s", (4, 20, 12), "float32"), ("conv", (2, 2 * 24 + 80), "float32")))
    assert needs[1] == StateNeed((("s", (2, 16, 20), "float32"),)) and needs[2] == StateNeed((("s", (3, 8, 12), "float32"),))
    assert needs[(3, 0)] != needs[(0, 0)]
    model = build_model(GIZU_2)
    assert dict(model.cache_needs())[(1, 1)] == StateNeed((("s", (3, 6, 10), "float32"),))  # one tap: nothing to keep


# --------------------------------------------------------------------------- the cache of a window that keeps first tokens
@pytest.mark.parametrize("window,keep", [(5, 1), (5, 4), (5, 5), (1, 9), (12, 3), (3, 30)])
def test_pages_of_the_first_tokens_outlive_the_window(window, keep):
    """Whatever the portions, every position that a later query can read lies on a page the request holds, and the others are
    given back; two requests on a pool that would not hold both in full."""
    P, total = 4, 61
    need = PagedKVNeed((("k", 1, 4),), window, keep)
    m = CacheManager([(0, need)], P, 64, 2, 64, torch.float32, torch.device("cpu"), poison=True, max_step_tokens=8)
    g = m.paged[0]
    assert g.pool.num_pages == 2 * (-(-(window + 8) // P) + 1 + -(-keep // P))
    rng = np.random.default_rng(window * 100 + keep)
    for rid in ("a", "b", "c"):
        m.open(rid)
        done = 0
        while done < total:
            n = int(min(rng.integers(1, 9), total - done))
            m.begin_step([(rid, n)])
            row = m.requests[rid].row
            for p in range(done, done + n):      # the step's queries
                for j in range(p + 1):
                    if p - j < window or j < keep:
                        assert g.table_host[row, j // P] != 0, (rid, p, j)
            m.end_step()
            m.check()
            done += n
            held = {b for b in range(g.width) if g.table_host[row, b]}
            first = max(0, done - window + 1)
            assert held == {b for b in range(-(-done // P)) if b >= first // P or b * P < keep}
            assert len(held) <= m.pages_to_admit(total)[0]
        if rid == "b":  # a step that does not run gives its pages back
            free = g.pool.free_count
            m.begin_step([(rid, 3)])
            m.abort_step()
            m.check()
            assert g.pool.free_count == free
        if rid != "a":
            m.close(rid)
            m.check()
    m.close("a")
    assert g.pool.free_count == g.pool.num_pages


@pytest.mark.parametrize("key_tile,rows", [(0, 16), (0, 64), (128, 128)])
@pytest.mark.parametrize("window,keep", [(40, 4), (9, 100), (200, 1), (1, 64), (65, 130)])
def test_work_lists_number_the_kept_tokens_and_the_window(key_tile, rows, window, keep):
    """Turned back into positions as the kernels do it, a tile's pieces cover what its queries read, each position once,
    and no more than a quantum before the window and behind the kept tokens."""
    q = key_tile or SPLIT_QUANTUM
    span = -(-keep // q) * q
    segs = [(1, 1), (70, 70), (2, 131), (1, 64), (33, 497), (1, 3000), (300, 1300)]
    for kw in (dict(), dict(fixed_splits=3), dict(sm_count=4096, min_split_keys=q)):
        plan = build_plan(segs, 2, rows, window, 1, key_tile=key_tile, keep_first=keep, **kw)
        tiles = {}
        for seg, tok0, ntok, b, e, n, i, base in plan.items.tolist():
            q_len, kv_len = segs[seg]
            lo = max(0, kv_len - q_len + tok0 - window + 1)
            jump = max(0, lo // q * q - span)
            assert b >= e or b % q == 0
            got = [v if v < span else v + jump for v in range(b, e)]
            tiles.setdefault((seg, tok0, ntok), []).extend(got)
        for (seg, tok0, ntok), got in tiles.items():
            q_len, kv_len = segs[seg]
            assert len(set(got)) == len(got)
            p0 = kv_len - q_len + tok0
            read = {j for p in range(p0, p0 + ntok) for j in list(range(max(0, p - window + 1), p + 1)) + list(range(min(keep, p + 1)))}
            assert read <= set(got)
            assert all(j < span or j > p0 - window - q for j in got) and max(got) == p0 + ntok - 1


# --------------------------------------------------------------------------- the plain mechanisms among themselves
def test_the_framework_and_the_plain_model_scale_frequencies_alike():
    from freetoken_b200.parts import BuildEnv, Workspace
    from freetoken_b200.parts.rope import InterleavedRope

    cpu = torch.device("cpu")
    for dims, base, bands in [(8, 100.0, (2.0, 1.0, 4.0, 64)), (32, 10000.0, (4.0, 1.0, 4.0, 256)), (64, 500000.0, (8.0, 1.0, 4.0, 8192)),
                              (16, 400.0, (16.0, 0.5, 2.0, 32)), (2, 10.0, (3.0, 1.0, 1.0, 7)), (12, 50.0, None)]:
        sc = None if bands is None else dict(zip(("factor", "low", "high", "original"), bands))
        want = plain_model.frequencies({"dims": dims, "base": base, "scaling": sc})
        env = BuildEnv(dtype=torch.float32, device=cpu, max_seq_len=40, max_step_tokens=1, workspace=Workspace(cpu))
        rope = InterleavedRope(PartSpec("rope_interleaved", dict(rotary_dim=dims, theta=base, precise=True, band_scaling=bands)), env)
        torch.testing.assert_close(rope.frequencies(), torch.tensor(want, dtype=torch.float64), rtol=1e-12, atol=0)
        torch.testing.assert_close(rope.table()[33, 0], torch.tensor(math.cos(33 * want[0])).float(), rtol=1e-6, atol=1e-6)
        plain = plain_model.frequencies({"dims": dims, "base": base})
        if bands is not None:
            assert all(f / bands[0] - 1e-12 <= g <= f + 1e-12 for f, g in zip(plain, want))
    assert plain_model.frequencies({"dims": 64, "base": 500000.0, "scaling": dict(factor=8.0, low=1.0, high=4.0, original=8192)})[0] == 1.0


def test_scaled_frequencies_in_their_three_bands():
    sc = dict(factor=8.0, low=1.0, high=4.0, original=100.0)
    f = plain_model.frequencies({"dims": 6, "base": (100.0 / 4) ** 1.5, "scaling": sc})
    raw = plain_model.frequencies({"dims": 6, "base": (100.0 / 4) ** 1.5})
    assert f[0] == raw[0]                                   # wavelength 2 pi < 25: kept
    assert raw[2] / f[2] == pytest.approx(8.0)              # wavelength over 100: divided
    wave = 2 * math.pi / raw[1]
    assert 25 < wave < 100
    s = (100.0 / wave - 1.0) / 3.0
    assert f[1] == pytest.approx((1 - s) * raw[1] / 8 + s * raw[1])


def test_the_two_pairings_are_one_rotation_of_reordered_columns():
    torch.manual_seed(0)
    f = [0.7, 0.11, 0.03]
    x = torch.randn(9, 2, 8).double()
    order = [0, 2, 4, 1, 3, 5, 6, 7]     # neighbours side by side -> halves
    torch.testing.assert_close(plain_model.rotate_halves(x[..., order], f), plain_model.rotate_neighbours(x, f)[..., order])
    torch.testing.assert_close(plain_model.rotate_neighbours(x, f)[..., 6:], x[..., 6:])
    q, k = torch.randn(6).double().expand(9, 1, 6), torch.randn(6).double().expand(9, 1, 6)
    s = plain_model.rotate_halves(q, f)[:, 0] @ plain_model.rotate_halves(k, f)[:, 0].T
    for i in range(8):
        torch.testing.assert_close(s[i + 1, i], s[1, 0])    # a score depends on the distance alone


def test_the_plain_window_keeps_its_first_tokens():
    v = plain_model.visible(8, 3, 2)
    assert v[7].tolist() == [True, True, False, False, False, True, True, True]
    assert v[1].tolist() == [True, True] + [False] * 6 and v[3].tolist() == [True] * 4 + [False] * 4
    assert torch.equal(plain_model.visible(5, None, 0), torch.ones(5, 5, dtype=torch.bool).tril())


def test_a_sink_is_a_key_without_a_value():
    s = torch.tensor([[1.0, 2.0, -math.inf]]).double()
    p = plain_model.softmax_with_sink(s, torch.tensor(0.5).double())
    whole = torch.softmax(torch.tensor([1.0, 2.0, 0.5]).double(), -1)
    torch.testing.assert_close(p[0], torch.tensor([float(whole[0]), float(whole[1]), 0.0]).double())


def test_the_plain_delta_rule_with_equal_decays_is_the_scalar_one():
    """With one decay for all channels the rule is the known gated delta rule; with beta 1, no decay and repeated unit keys the
    state holds the last value written under a key; a channel that decays forgets only its own share."""
    torch.manual_seed(1)
    T, D, Dv = 12, 4, 3
    q, k, v = torch.randn(T, D).double(), torch.nn.functional.normalize(torch.randn(T, D).double(), dim=-1), torch.randn(T, Dv).double()
    beta, g = torch.rand(T).double(), torch.rand(T).double()
    S = torch.zeros(D, Dv).double()
    want = []
    for t in range(T):  # the other way round: the correction as a product from the left
        S = (torch.eye(D).double() - beta[t] * torch.outer(k[t], k[t])) @ (g[t] * S) + beta[t] * torch.outer(k[t], v[t])
        want.append(q[t] @ S)
    torch.testing.assert_close(plain_model.delta_rule(q, k, v, beta, g[:, None].expand(T, D)), torch.stack(want))
    e = torch.eye(D).double()
    ones = torch.ones(T).double()
    decay = torch.ones(T, D).double()
    decay[:, 1] = 0.5
    o = plain_model.delta_rule(e[[0, 1, 0, 1]], e[[0, 1, 2, 3]], v[:4], ones, decay)
    torch.testing.assert_close(o, torch.stack([v[0], v[1], v[0], 0.25 * v[1]]))


def test_plain_retention_is_a_sum_over_the_past():
    torch.manual_seed(2)
    m = dict(heads=2, dim=4, vdim=3, decay=[0.9, 0.5], rot={"dims": 4, "base": 50.0})
    w = {n: torch.randn(r, 6).double() for n, r in (("q", 8), ("k", 8), ("v", 6), ("g", 6))}
    w["o"] = torch.eye(6).double()
    h = torch.randn(7, 6).double()
    got = plain_model.retention(h, w, m, 1e-5)
    f = plain_model.frequencies(m["rot"])
    q, k = (plain_model.rotate_halves((h @ w[n].T).view(7, 2, 4), f) for n in "qk")
    v = (h @ w["v"].T).view(7, 2, 3)
    gate = plain_model.silu(h @ w["g"].T).view(7, 2, 3)
    for a, d in enumerate(m["decay"]):
        i = torch.arange(7)
        weight = torch.where(i[:, None] >= i[None, :], torch.tensor(d).double() ** (i[:, None] - i[None, :]).clamp(min=0), 0.0)
        o = ((q[:, a] @ k[:, a].T) / 2.0 * weight) @ v[:, a]
        torch.testing.assert_close(got.view(7, 2, 3)[:, a], plain_model.over_rms(o, 1e-5) * gate[:, a])


def test_plain_experts_come_from_the_best_groups():
    s = torch.tensor([[0.05, 0.30, 0.25, 0.01, 0.20, 0.19], [0.3, 0.1, 0.15, 0.15, 0.2, 0.1]]).double()
    chosen, gap = plain_model.choose_experts(s, 2, 3, 2)           # groups (0, 1), (2, 3), (4, 5)
    assert chosen.tolist() == [[1, 2], [0, 4]]
    assert gap[0] == pytest.approx(0.05) and gap[1] == pytest.approx(0.05)
    chosen, _ = plain_model.choose_experts(s, 2, 3, 1)             # one group: its second best, however small
    assert chosen.tolist() == [[1, 0], [0, 1]]
    chosen, _ = plain_model.choose_experts(s, 3, 1, 1)
    assert chosen.tolist() == [[1, 2, 4], [0, 4, 2]]
    torch.manual_seed(3)
    w = {f"e{e}.{n}": torch.randn(*z).double() for e in range(4) for n, z in (("gate", (5, 6)), ("up", (5, 6)), ("down", (6, 5)))}
    w["router"] = torch.randn(4, 6).double()
    h = torch.randn(3, 6).double()
    out = plain_model.mixture(h, w, {"router": {"experts": 4, "top": 4, "groups": {"count": 2, "keep": 2}}})
    s = torch.softmax(h @ w["router"].T, -1)                       # every expert, by its score as it is
    want = sum(s[:, e, None] * plain_model.gated_layer(h, w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"]) for e in range(4))
    torch.testing.assert_close(out, want)


# --------------------------------------------------------------------------- the engine on CPU stand-ins
@pytest.mark.parametrize("name", ["G1", "G2", "G3", "G4", "G5"])
def test_cuts_agree_with_the_plain_model(name, tmp_path_factory, cpu_ops):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainGizulorn(folder)
    toks = tokens_for(plain.vocab, 41, 7)
    want = plain.logits(toks)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=30)
    torch.testing.assert_close(replay_whole(eng, "w", toks), want, **TOL)
    torch.testing.assert_close(replay_cuts(eng, "c", toks, [5, 2, 11, 2, 3, 7]), want, **TOL)
    torch.testing.assert_close(replay_cuts(eng, "o", toks[:24], []), want[:24], **TOL)
    eng.cache.check()
    assert all(g.pool.free_count == g.pool.num_pages for g in eng.cache.paged)


@pytest.mark.parametrize("name", ["G1", "G4"])
def test_batches_of_unequal_requests_and_slots_used_again(name, tmp_path_factory, cpu_ops):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainGizulorn(folder)
    lengths = {"r0": 25, "r1": 33, "r2": 18, "r3": 29, "r4": 21, "r5": 27}
    seqs = {r: tokens_for(plain.vocab, n, i) for i, (r, n) in enumerate(lengths.items())}
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=4 * 10, max_step=40)
    got = replay_mixed(eng, seqs, mixed_schedule(lengths, seed=5))
    for r, toks in seqs.items():
        torch.testing.assert_close(got[r], plain.logits(toks), **TOL, msg=lambda m: f"{r}: {m}")
    assert eng.cache.slots.free_count == 4
    assert any(g.pool.handed_out > g.pool.num_pages for g in eng.cache.paged)


def test_a_slot_used_again_starts_from_nothing(tmp_path_factory, cpu_ops):
    """One request slot: every request gets the slot (and pages) of the one before; what the states and convolutions of the
    earlier owner left must not leak."""
    folder = model_folder(tmp_path_factory.getbasetemp(), "G1", GIZU_1)
    plain = PlainGizulorn(folder)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=12, reqs=1, max_step=24)
    for i in range(3):
        toks = tokens_for(plain.vocab, 20 + i, 30 + i)
        torch.testing.assert_close(replay_cuts(eng, f"r{i}", toks, [1, 1, 6, 2]), plain.logits(toks), **TOL)


@pytest.mark.parametrize("name", ["G1", "G2"])
def test_the_stream_after_every_layer_is_the_plain_models(name, tmp_path_factory, cpu_ops):
    from freetoken_b200.parts.base import StreamSum, as_rows

    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainGizulorn(folder)
    toks = tokens_for(plain.vocab, 19, 2)
    want = plain.layer_sums(toks)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=30)
    seen = []
    for b in eng.model.blocks:
        def wrapped(x, residual, step, cache, writes, orig=b.forward):
            y = orig(x, residual, step, cache, writes)
            after = residual.clone()
            rest = as_rows(y, None, after)  # what the layer leaves to the next one's first kernel
            if rest is not None:
                StreamSum.of(rest).fold(after)
            seen.append(after)
            return y

        b.forward = wrapped
    eng.step([StepEntry("a", toks, [len(toks) - 1])])
    assert len(seen) == len(want)
    for i, (s, w) in enumerate(zip(seen, want)):
        torch.testing.assert_close(s, w, **TOL, msg=lambda m: f"after layer {i}: {m}")


def test_a_planted_mistake_in_the_plain_model_shows(tmp_path_factory, cpu_ops):
    """The comparisons above notice each mechanism: with one of them changed in the plain model its logits move by
    hundreds of times the tolerance."""
    folder = model_folder(tmp_path_factory.getbasetemp(), "G1", GIZU_1)
    plain = PlainGizulorn(folder)
    toks = tokens_for(plain.vocab, 30, 4)
    want = plain.logits(toks)

    def moved(change):
        other = PlainGizulorn(folder)
        other.raw = copy.deepcopy(other.raw)
        change(other)
        return float((other.logits(toks) - want).abs().max())

    def with_config(path, value):
        def change(o):
            d = o.raw
            for k in path[:-1]:
                d = d[k]
            d[path[-1]] = value
        return change

    def put(name, value):
        def change(o):
            o.w[name] = torch.full_like(o.w[name], value)
        return change

    left = ["layers", 0, "mixer", "left"]
    assert moved(lambda o: None) == 0.0
    for what, change in [
        ("window", with_config(left + ["mask", "size"], 10)), ("kept tokens", with_config(left + ["mask", "keep_first"], 2)),
        ("scaled frequencies", with_config(left + ["rot", "scaling"], None)), ("rotated dimensions", with_config(left + ["rot", "dims"], 10)),
        ("sink", put("l0.mix.left.sink", -50.0)), ("left factor", with_config(["layers", 0, "mixer", "left_scale"], 1.0)),
        ("right factor", with_config(["layers", 0, "mixer", "right_scale"], 1.0)), ("decay per channel", put("l0.mix.right.a2", 0.0)),
        ("decay bias", put("l0.mix.right.dt_bias", 0.0)), ("step size", put("l0.mix.right.b", 0.0)),
        ("gate", put("l0.mix.right.g2", 0.0)), ("convolution", put("l0.mix.right.k.conv", 0.0)),
        ("retention's decay", with_config(["layers", 2, "mixer", "decay"], [0.9, 0.99, 0.9])),
        ("retention's rotation", with_config(["layers", 1, "mixer", "rot"], None)),
        ("groups", with_config(["layers", 2, "mlp", "router", "groups"], {"count": 1, "keep": 1})),
        ("shared gate", put("l0.mlp.shared.sg", 0.0)),
    ]:
        assert moved(change) > 100 * TOL["atol"], what


def test_retention_keeps_its_first_token_for_long(cpu_ops, tmp_path_factory):
    """G4's second layer has a head that forgets nothing and one that forgets at once: long sequences in portions."""
    folder = model_folder(tmp_path_factory.getbasetemp(), "G4", GIZU_4)
    plain = PlainGizulorn(folder)
    toks = tokens_for(plain.vocab, 150, 8)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=48)
    torch.testing.assert_close(replay_cuts(eng, "a", toks, [65, 64, 2, 11]), plain.logits(toks), **TOL)


def test_a_model_cut_to_its_first_layers():
    assert len(architecture_of(GIZU_1).parse_config(GIZU_1, num_layers=2).layers) == 2


def test_a_pair_with_factors_takes_two_branches():
    from freetoken_b200.parts import MIXERS, BuildEnv, Workspace

    cpu = torch.device("cpu")
    env = BuildEnv(dtype=torch.float32, device=cpu, max_seq_len=8, max_step_tokens=8, workspace=Workspace(cpu))
    branch = ("left", PartSpec("retention", dict(hidden=8, n_heads=1, head_dim=4, decay=(0.5,))))
    with pytest.raises(ConfigError):
        MIXERS.build(PartSpec("side_by_side", dict(hidden=8, branches=(branch,), scales=(1.0,))), env)
    with pytest.raises(ConfigError):
        MIXERS.build(PartSpec("retention", dict(hidden=8, n_heads=2, head_dim=4, decay=(0.5,))), env)


def plain_for_the_command_line(folder):
    from types import SimpleNamespace

    plain = PlainGizulorn(folder)
    return SimpleNamespace(cfg=SimpleNamespace(vocab=plain.vocab), logits=lambda toks: plain.logits(toks).float())


def test_the_command_line_makes_a_model_generates_and_replays(tmp_path, capsys, cpu_ops):
    from test_cli import generate_and_replay, make_model

    folder = make_model(tmp_path, GIZU_1, capsys)
    generate_and_replay(folder, "cpu", "float32", capsys, tmp_path, plain_for_the_command_line(folder))
