"""Vodatar without a GPU: its config reader, model description and checkpoint names, the plain statements of its
mechanisms against other ways of writing them, and the engine's step, cache, state and batching logic with the plain
PyTorch statements of the kernels (tests/kernel_refs.py) standing in for the CUDA kernels."""

import copy
import math

import pytest
import torch

import kernel_refs
from helpers import make_engine, mixed_schedule, model_folder, replay_cuts, replay_mixed, replay_whole, tokens_for
from plain import vodatar_plain as plain_model
from plain.vodatar_plain import PlainVodatar
from tiny_vodatar import ALL, PAGE, VODA_1, VODA_2, VODA_3, VODA_4

from freetoken_b200.config.spec import PagedKVNeed, StateNeed
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
    _, cfg, spec, expected = describe_model(VODA_1)
    assert [l.mixer.kind for l in spec.layers] == ["differential_attention", "latent_attention"] * 2
    assert [l.ffn.kind for l in spec.layers] == ["moe", "none", "moe", "moe"]
    assert all(l.block.kind == "gated_sandwich_residual" and (l.block["groups"], l.block["taps"], l.block["mult"]) == (2, 4, 0.6)
               for l in spec.layers)
    assert [(e.layer, e.add_pass_vector, e.mix_embedding, e.cache_from) for e in spec.schedule] == [
        (0, None, False, None), (1, 0, True, None), (2, None, False, None), (1, 1, True, None), (2, None, False, None),
        (3, None, False, None)]
    a = spec.layers[0].mixer
    assert (a["head_dim"], a["v_head_dim"], a["taps"], a["softcap"], a["diff"], a["scale"]) == (8, 20, 3, 9.0, 0.2, 0.4)
    assert a["position"].kind == "rope_interleaved" and a["position"]["yarn"] is None
    b = spec.layers[1].mixer
    assert (b["q_rank"], b["kv_rank"], b["rot_dim"], b["sink"], b["window"]) == (None, 20, 8, None, None)
    assert b["position"]["yarn"] == (2.0, 64.0, 8.0, 1.0) and b["position"]["rotary_dim"] == 8
    f = spec.layers[2].ffn
    assert (f["n_experts"], f["identity"], f["top_k"], f["shared_inter"], f["shared_gate"], f["scoring"]) == (5, 1, 3, 32, True, "softmax")
    assert spec.embedding["norm"]["groups"] == 2 and spec.final_norm["groups"] == 2
    assert expected["l0.mix.qkv_proj.weight"].shape == (4 * 16 + 2 * 16 + 2 * 20, 64)
    assert expected["l0.mix.conv.weight"].shape == (4 * 16 + 2 * 16 + 2 * 20, 3)
    assert expected["l0.mlp.gate.weight"].shape == (8, 64) and expected["l0.mlp.e_score_correction_bias"].shape == (8,)
    assert expected["l0.mlp.experts.down_proj"].shape == (6, 64, 40) and expected["l0.mlp.shared_gate.weight"].shape == (1, 64)
    assert expected["loop.in.weight"].shape == (64, 128) and expected["loop.step"].shape == (2, 64)
    assert expected["l0.canon2"].shape == (64, 4) and expected["l0.rg1"].shape == (64, 64) and expected["l0.rg2.b"].shape == (64,)
    assert not any(n in expected for n in ("l1.norm2", "l1.canon2", "l1.rg2"))
    _, _, spec4, expected4 = describe_model(VODA_4)
    assert spec4.pass_input is None and spec4.pass_vectors is None and "loop.in.weight" not in expected4
    assert "l0.mlp.shared_gate.weight" not in expected4 and "l1.mlp.shared_gate.weight" in expected4
    assert not describe_model(VODA_2)[2].layers[1].mixer["softcap"]


def test_the_checkpoint_names_are_the_designs():
    arch, cfg, _, _ = describe_model(VODA_1)
    rules = arch.fusion_rules(cfg)
    sources = {s for r in rules for s in r.sources}
    for name in ("embed", "embed.norm", "head", "final.norm", "loop.in", "l0.mix.q", "l0.mix.k.conv", "l0.mix.o", "l1.mix.dkv",
                 "l1.mix.dkv.norm", "l1.mix.uk", "l1.mix.uv", "l1.mix.q", "l0.mlp.e5.down", "l0.mlp.router", "l0.mlp.correction",
                 "l0.mlp.shared.up", "l0.mlp.shared.sg"):
        assert name in sources, name
    assert not any("e6." in s for s in sources if s.startswith("l0."))  # identity experts have no tensors


def test_written_folders_hold_the_designs_tensors(tmp_path_factory):
    from freetoken_b200.weights.safetensors_io import ModelFolder

    mf = ModelFolder(model_folder(tmp_path_factory.getbasetemp(), "V1", VODA_1))
    names = set(mf.names())
    for n in ("loop.in", "loop.step", "l0.rg1", "l0.rg1.b", "l0.canon1", "l0.norm1b", "l0.mix.lq1", "l0.mix.lk2", "l0.mix.v.conv"):
        assert n in names, n
    assert {mf.dtype(n) for n in names} == {torch.bfloat16}


def test_config_errors_name_the_key():
    def broken(path, value, delete=False):
        raw = copy.deepcopy(VODA_1)
        d = raw
        for k in path[:-1]:
            d = d[k]
        if delete:
            del d[path[-1]]
        else:
            d[path[-1]] = value
        return raw

    for raw, word in [
        (broken(["vocab"], None, True), "vocab"),
        (broken(["norm", "groups"], 3), "norm.groups"),
        (broken(["norm", "eps"], None, True), "eps"),
        (broken(["canon", "taps"], 17), "taps"),
        (broken(["residual_mult"], None, True), "residual_mult"),
        (broken(["loop", "stop"], 5), "loop"),
        (broken(["loop", "times"], 0), "loop"),
        (broken(["layers", 0, "mixer", "kv_heads"], 3), "kv_heads"),
        (broken(["layers", 0, "mixer", "diff"], None, True), "diff"),
        (broken(["layers", 0, "mixer", "softcap"], -1.0), "softcap"),
        (broken(["layers", 0, "mixer", "rot", "dims"], 10), "rot.dims"),
        (broken(["layers", 0, "mixer", "conv"], 0), "conv"),
        (broken(["layers", 1, "mixer", "kv_rank"], None, True), "kv_rank"),
        (broken(["layers", 1, "mixer", "rot", "scaling", "fast"], None, True), "fast"),
        (broken(["layers", 0, "mlp", "kind"], "dense"), "kind"),
        (broken(["layers", 0, "mlp", "router", "top"], 9), "router.top"),
        (broken(["layers", 2, "type"], "conv"), "type"),
    ]:
        with pytest.raises(ConfigError, match=word):
            architecture_of(raw).parse_config(raw)


def test_pages_and_states_are_each_pass_own():
    model = build_model(VODA_1)
    needs = dict(model.cache_needs())
    rows = 4 * 16 + 2 * 16 + 2 * 20
    assert needs[(0, 0)] == PagedKVNeed((("k", 2, 32), ("v", 2, 32)), None)  # two maps of 8, values of 20: rows of 32
    assert needs[(0, 1)] == StateNeed((("conv", (2, rows), "float32"),))
    assert needs[1] == needs[3] == PagedKVNeed((("kv", 1, 32),), None)       # layer 1, in both passes
    assert needs[(2, 1)] == needs[(4, 1)]
    blocks = dict(model.block_state_needs())
    assert sorted(blocks) == [0, 1, 2, 3, 4, 5]
    assert blocks[1] == StateNeed((("conv1", (3, 64), "float32"),))          # no feed-forward: one convolution
    assert blocks[5] == StateNeed((("conv1", (3, 64), "float32"), ("conv2", (3, 64), "float32")))
    model2 = build_model(VODA_2)
    assert not any(isinstance(n, StateNeed) for _, n in model2.cache_needs()) and not model2.block_state_needs()


# --------------------------------------------------------------------------- the plain mechanisms among themselves
def test_the_plain_norm_takes_each_group_alone():
    x = torch.tensor([[3.0, 4.0, 0.6, 0.8]], dtype=torch.float64)
    w = torch.tensor([1.0, 1.0, 2.0, 1.0], dtype=torch.float64)
    y = plain_model.group_norm(x, w, 2, 0.0)
    f = math.sqrt(12.5)
    torch.testing.assert_close(y[0], torch.tensor([3 / f, 4 / f, 2 * 3 / f, 4 / f], dtype=torch.float64))
    torch.testing.assert_close(plain_model.group_norm(x, w, 1, 0.25), plain_model.unit(x, 0.25) * w)


def test_the_plain_convolution_reads_backwards_only():
    x = torch.arange(8.0).view(4, 2)
    w = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]])
    c = plain_model.causal_conv(x, w)
    assert c[0].tolist() == [0.0, 1.0] and c[2].tolist() == [0.0 + 10 * 2.0 + 100 * 4.0, 5.0]
    assert plain_model.causal_conv(x[:1], w).tolist() == [[0.0, 1.0]]


def test_the_framework_and_the_plain_model_stretch_frequencies_alike():
    from freetoken_b200.parts import BuildEnv, Workspace
    from freetoken_b200.parts.rope import InterleavedRope
    from freetoken_b200.config.spec import PartSpec

    cpu = torch.device("cpu")
    for dims, base, yarn in [(8, 100.0, (2.0, 64, 8.0, 1.0)), (32, 10000.0, (4.0, 256, 32.0, 1.0)), (16, 400.0, (16.0, 32, 2.0, 0.25)),
                             (64, 500000.0, (8.0, 4096, 32.0, 1.0)), (4, 50.0, (3.0, 128, 4.0, 0.5)), (2, 10.0, (2.0, 7, 3.0, 2.9))]:
        want = plain_model.yarn_frequencies(dims, base, *yarn)
        env = BuildEnv(dtype=torch.float32, device=cpu, max_seq_len=40, max_step_tokens=1, workspace=Workspace(cpu))
        rope = InterleavedRope(PartSpec("rope_interleaved", dict(rotary_dim=dims, theta=base, precise=True, yarn=yarn)), env)
        torch.testing.assert_close(rope.frequencies(), torch.tensor(want, dtype=torch.float64), rtol=1e-12, atol=0)
        mag = 0.1 * math.log(yarn[0]) + 1.0
        tab = rope.table()
        torch.testing.assert_close(tab[33, 0], torch.tensor(math.cos(33 * want[0]) * mag).float(), rtol=1e-6, atol=1e-6)
        torch.testing.assert_close(tab[33, dims // 2], torch.tensor(math.sin(33 * want[0]) * mag).float(), rtol=1e-6, atol=1e-6)
        plain = plain_model.plain_frequencies(dims, base)
        assert all(f / yarn[0] - 1e-12 <= g <= f + 1e-12 for f, g in zip(plain, want))


def test_the_plain_rotation_turns_neighbours_and_keeps_distances():
    torch.manual_seed(0)
    f = [0.7, 0.11]
    q, k = torch.randn(1, 6).double().expand(9, 6), torch.randn(1, 6).double().expand(9, 6)
    rq, rk = plain_model.rotate_neighbours(q, f), plain_model.rotate_neighbours(k, f)
    s = rq @ rk.T
    for i in range(8):
        for j in range(8):
            torch.testing.assert_close(s[i + 1, j + 1], s[i, j])      # a score depends on the distance alone
    torch.testing.assert_close(rq[:, 4:], q[:, 4:])                   # columns behind the rotated ones stay
    torch.testing.assert_close(plain_model.rotate_neighbours(q, f, 1.5)[:, :4], 1.5 * rq[:, :4])


def test_the_plain_differential_attention_is_two_attentions():
    """With lambda made 0 (its three terms cancel) the second map does not matter; with the maps equal the output is the
    plain attention's scaled by 1 - lambda before the norm, which the norm takes out again (up to the sign)."""
    torch.manual_seed(1)
    m = dict(heads=2, kv_heads=1, dim=4, vdim=6, scale=0.5, softcap=3.0, diff=0.3, rot={"dims": 4, "base": 100.0})
    W = 10
    w = {n: torch.randn(r, W).double() / 3 for n, r in (("q", 16), ("k", 8), ("v", 6))}
    w.update({n + ".conv": torch.randn(w[n].shape[0], 3).double() for n in ("q", "k", "v")})
    w["o"] = torch.randn(W, 12).double()
    zero = torch.zeros(4).double()
    for n in ("lq1", "lk1", "lq2", "lk2"):
        w[n] = zero.clone()
    h = torch.randn(7, W).double()
    # exp(0) - exp(x) + diff = 0 for x = ln(1 + diff)
    w["lq2"][0], w["lk2"][0] = 1.0, math.log(1.3)
    one = plain_model.differential_attention(h, w, m, 1e-9)
    other = dict(w, q=w["q"].clone(), k=w["k"].clone())
    other["q"].view(2, 2, 4, W)[:, 1] = torch.randn(2, 4, W).double()
    torch.testing.assert_close(plain_model.differential_attention(h, other, m, 1e-9), one)
    w["lq2"] = zero.clone()  # lambda = 0.3: now it does
    assert float((plain_model.differential_attention(h, dict(other, lq2=zero), m, 1e-9)
                  - plain_model.differential_attention(h, w, m, 1e-9)).abs().max()) > 1e-2


def test_the_plain_mixture_hands_the_input_back_for_identity_experts():
    torch.manual_seed(2)
    W = 6
    w = {f"e{e}.{n}": torch.randn(*s).double() for e in range(2) for n, s in (("gate", (4, W)), ("up", (4, W)), ("down", (W, 4)))}
    w["router"], w["correction"] = torch.randn(4, W).double(), torch.tensor([-9.0, -9.0, 9.0, 8.0]).double()
    m = {"router": {"experts": 2, "identity": 2, "top": 2}}
    h = torch.randn(5, W).double()
    torch.testing.assert_close(plain_model.mixture(h, w, m), h)  # both chosen experts are identities: weights add up to 1
    w["correction"] = torch.zeros(4).double()
    chosen, weights, _ = plain_model.choose_experts(h, w["router"], torch.tensor([0.0, 0.0, 5.0, 0.0]).double(), 2)
    s = torch.softmax(h @ w["router"].T, -1)
    assert (chosen[:, 0] == 2).all()  # the correction decides the choice ...
    torch.testing.assert_close(weights[:, 0], s[:, 2] / s.gather(-1, chosen).sum(-1))  # ... and not the weight


def test_the_plain_passes():
    assert PlainVodatar(raw=VODA_1, weights={}).passes() == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert PlainVodatar(raw=VODA_3, weights={}).passes() == [(0, 0), (1, None), (0, 1), (1, None), (0, 2), (1, None)]
    assert PlainVodatar(raw=VODA_4, weights={}).passes() == [(0, None), (1, None), (2, None)]


# --------------------------------------------------------------------------- the engine on CPU stand-ins
@pytest.mark.parametrize("name", ["V1", "V2", "V3", "V4"])
def test_cuts_agree_with_the_plain_model(name, tmp_path_factory, cpu_ops):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainVodatar(folder)
    toks = tokens_for(plain.vocab, 41, 7)
    want = plain.logits(toks)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=30)
    torch.testing.assert_close(replay_whole(eng, "w", toks), want, **TOL)
    torch.testing.assert_close(replay_cuts(eng, "c", toks, [5, 2, 11, 2, 3, 7]), want, **TOL)
    torch.testing.assert_close(replay_cuts(eng, "o", toks[:12], []), want[:12], **TOL)
    eng.cache.check()
    assert all(g.pool.free_count == g.pool.num_pages for g in eng.cache.paged)


def test_batches_of_unequal_requests_and_slots_used_again(tmp_path_factory, cpu_ops):
    folder = model_folder(tmp_path_factory.getbasetemp(), "V1", VODA_1)
    plain = PlainVodatar(folder)
    lengths = {"r0": 25, "r1": 33, "r2": 18, "r3": 29, "r4": 21, "r5": 27}
    seqs = {r: tokens_for(plain.vocab, n, i) for i, (r, n) in enumerate(lengths.items())}
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=4 * 10)
    got = replay_mixed(eng, seqs, mixed_schedule(lengths, seed=5))
    for r, toks in seqs.items():
        torch.testing.assert_close(got[r], plain.logits(toks), **TOL, msg=lambda m: f"{r}: {m}")
    assert eng.cache.slots.free_count == 4
    for g in eng.cache.paged:
        assert g.pool.handed_out > g.pool.num_pages


def test_a_slot_used_again_starts_from_nothing(tmp_path_factory, cpu_ops):
    """One request slot: every request gets the slot (and pages) of the one before; what the convolutions of the earlier
    owner left must not leak, in any pass."""
    folder = model_folder(tmp_path_factory.getbasetemp(), "V4", VODA_4)
    plain = PlainVodatar(folder)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=12, reqs=1)
    for i in range(3):
        toks = tokens_for(plain.vocab, 20 + i, 30 + i)
        torch.testing.assert_close(replay_cuts(eng, f"r{i}", toks, [1, 1, 6, 2]), plain.logits(toks), **TOL)


@pytest.mark.parametrize("name", ["V1", "V4"])
def test_the_stream_after_every_layer_run_is_the_plain_models(name, tmp_path_factory, cpu_ops):
    folder = model_folder(tmp_path_factory.getbasetemp(), name, ALL[name])
    plain = PlainVodatar(folder)
    toks = tokens_for(plain.vocab, 19, 2)
    want = plain.layer_sums(toks)
    eng = make_engine(folder, "float32", "cpu", PAGE, pages=30)
    seen = []
    for b in set(eng.model.blocks):
        def wrapped(x, residual, step, cache, writes, orig=b.forward):
            y = orig(x, residual, step, cache, writes)
            after = residual.clone()
            y.fold(after)  # what the layer leaves to the next one's first kernel
            seen.append(after)
            return y

        b.forward = wrapped
    eng.step([StepEntry("a", toks, [len(toks) - 1])])
    assert len(seen) == len(want) == len(eng.spec.schedule)
    for i, (s, w) in enumerate(zip(seen, want)):
        torch.testing.assert_close(s, w, **TOL, msg=lambda m: f"after layer run {i}: {m}")


def test_a_planted_mistake_in_the_plain_model_shows(tmp_path_factory, cpu_ops):
    """The comparisons above notice each mechanism: with one of them left out of the plain model its logits move by
    hundreds of times the tolerance."""
    folder = model_folder(tmp_path_factory.getbasetemp(), "V1", VODA_1)
    plain = PlainVodatar(folder)
    toks = tokens_for(plain.vocab, 30, 4)
    want = plain.logits(toks)

    def moved(change):
        other = PlainVodatar(folder)
        change(other)
        return float((other.logits(toks) - want).abs().max())

    def with_config(path, value):
        def change(o):
            o.raw = copy.deepcopy(o.raw)
            d = o.raw
            for k in path[:-1]:
                d = d[k]
            d[path[-1]] = value
        return change

    def zero(name):
        def change(o):
            o.w[name] = torch.zeros_like(o.w[name])
        return change

    assert moved(lambda o: None) == 0.0
    for what, change in [
        ("soft cap", with_config(["layers", 0, "mixer", "softcap"], None)),
        ("stretched frequencies", with_config(["layers", 1, "mixer", "rot", "scaling"], None)),
        ("second map", with_config(["layers", 0, "mixer", "diff"], 0.0)),
        ("input convolution", zero("l0.canon1")), ("second input convolution", zero("l2.canon2")),
        ("gate bias", zero("l0.rg1.b")), ("pass vector", zero("loop.step")), ("shared gate", zero("l0.mlp.shared.sg")),
        ("correction", zero("l0.mlp.correction")),
        ("norm groups", lambda o: setattr(o, "groups", 1)), ("factor", lambda o: setattr(o, "mult", 1.0)),
    ]:
        assert moved(change) > 100 * TOL["atol"], what


def test_a_model_cut_to_its_first_layers_keeps_what_is_left_of_the_loop():
    arch = architecture_of(VODA_1)
    cut = arch.parse_config(VODA_1, num_layers=2)
    assert len(cut.layers) == 2 and (cut.loop.start, cut.loop.stop) == (1, 2)


def plain_for_the_command_line(folder):
    from types import SimpleNamespace

    plain = PlainVodatar(folder)
    return SimpleNamespace(cfg=SimpleNamespace(vocab=plain.vocab), logits=lambda toks: plain.logits(toks).float())


def test_the_command_line_makes_a_model_generates_and_replays(tmp_path, capsys, cpu_ops):
    from test_cli import generate_and_replay, make_model

    folder = make_model(tmp_path, VODA_1, capsys)
    generate_and_replay(folder, "cpu", "float32", capsys, tmp_path, plain_for_the_command_line(folder))
