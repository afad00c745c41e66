"""Vodatar: from its typed config to a model description, and its checkpoint names.

Layers are ``gated_sandwich_residual`` blocks (norms over groups of channels on both sides of every sub-layer, a short
convolution in front of it, an element-wise gate and a constant factor behind it).  The mixer is
``differential_attention`` (convolved projections, interleaved rotation, soft-capped scores) or ``latent_attention`` (no
query latent, no gate; interleaved rotation with stretched frequencies).  The feed-forward is ``moe`` with a softmax router
whose correction counts for the choice only, identity experts and a gated shared expert, or none.  The embedding rows pass
a norm of their own.  A range of layers is repeated as schedule entries with caches and states of their own; each pass
starts with ``stream_mix`` (a product of the stream and the embedding output) and a vector of the pass.

Checkpoint names: ``embed``, ``embed.norm``, ``head``, ``final.norm``, ``loop.in``, ``loop.step`` and, per layer ``l<i>``:
``norm1``, ``norm1b``, ``norm2``, ``norm2b``, ``canon1``, ``canon2``, ``rg1``, ``rg1.b``, ``rg2``, ``rg2.b``; attention
``mix.{q,k,v}`` (each with ``.conv``), ``mix.{lq1,lk1,lq2,lk2,o}``; latent attention ``mix.{q,dkv,dkv.norm,uk,uv,o}``;
``mlp.e<j>.{gate,up,down}``, ``mlp.router``, ``mlp.correction``, ``mlp.shared.{gate,up,down,sg}``.  The projections of a
mixer's input are concatenated into one matrix; gate/up pairs and experts are stacked as for every other architecture here.
The reference has no such design.
"""

from __future__ import annotations

from typing import Any, List, Mapping, Optional

from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..config.vodatar import ARCHITECTURES, MAX_POSITION, VodatarConfig, VodatarRotation
from ..registry import Architecture, register_architecture
from ..weights.binder import FusionRule


def _position(rot: Optional[VodatarRotation]) -> PartSpec:
    if rot is None:
        return PartSpec("none")
    return PartSpec("rope_interleaved", dict(rotary_dim=rot.dims, theta=rot.base, precise=True, yarn=rot.yarn))


def schedule_of(cfg: VodatarConfig) -> List[ScheduleEntry]:
    """The order layers run in; every entry owns its cache and states."""
    L = len(cfg.layers)
    if cfg.loop is None:
        return [ScheduleEntry(i) for i in range(L)]
    a, b = cfg.loop.start, cfg.loop.stop
    out = [ScheduleEntry(i) for i in range(a)]
    for t in range(cfg.loop.times):
        out += [ScheduleEntry(i, add_pass_vector=t if i == a else None, mix_embedding=i == a) for i in range(a, b)]
    return out + [ScheduleEntry(i) for i in range(b, L)]


def build_spec(cfg: VodatarConfig) -> ModelSpec:
    W = cfg.width
    # random models: spreads that keep every activation of order one, so that a fault anywhere shows in the logits
    w_in = W ** -0.5
    norm = PartSpec("rmsnorm", dict(size=W, eps=cfg.norm_eps, gemma=False, groups=cfg.norm_groups))
    block = PartSpec("gated_sandwich_residual", dict(hidden=W, groups=cfg.norm_groups, eps=cfg.norm_eps, taps=cfg.canon_taps,
                                                     mult=cfg.residual_mult, init_std=w_in))
    layers: List[LayerSpec] = []
    for i, l in enumerate(cfg.layers):
        a = l.mixer
        if l.type == "attention":
            mixer = PartSpec("differential_attention", dict(
                hidden=W, n_heads=a.heads, n_kv_heads=a.kv_heads, head_dim=a.dim, v_head_dim=a.vdim, taps=a.taps,
                position=_position(a.rot), scale=a.scale, softcap=a.softcap, diff=a.diff, eps=cfg.norm_eps,
                init_std=(w_in, (a.heads * a.vdim) ** -0.5)))
        else:
            mixer = PartSpec("latent_attention", dict(
                hidden=W, n_heads=a.heads, head_dim=a.dim, rot_dim=a.rot_dim, v_head_dim=a.vdim, q_rank=None,
                kv_rank=a.kv_rank, eps=cfg.norm_eps, position=_position(a.rot), window=None, scale=a.scale, sink=None,
                init_std=(w_in, w_in, a.kv_rank ** -0.5, (a.heads * a.vdim) ** -0.5)))
        f = l.mlp
        if f is None:
            ffn = PartSpec("none")
        else:
            ffn = PartSpec("moe", dict(hidden=W, inter=f.ff, n_experts=f.experts, identity=f.identity, top_k=f.top,
                                       scoring="softmax", bias=True, scale=1.0, act="silu", shared_inter=f.shared_ff,
                                       shared_gate=bool(f.shared_ff), router_store="bfloat16", bias_std=0.05,
                                       init_std=(w_in, f.ff ** -0.5)))
        layers.append(LayerSpec(name=f"l{i}", block=block, mixer=mixer, ffn=ffn, mixer_name="mix", ffn_name="mlp"))
    looped = cfg.loop is not None
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=W, layers=tuple(layers),
        schedule=tuple(schedule_of(cfg)),
        embedding=PartSpec("token_embedding", dict(vocab=cfg.vocab, hidden=W, init_std=1.0, norm=norm)),
        final_norm=norm,
        head=PartSpec("linear_head", dict(tied=False, init_std=w_in)),
        max_position=MAX_POSITION,
        embedding_name="embed_tokens", final_norm_name="final.norm", head_name="head",
        pass_vectors=PartSpec("pass_vectors", dict(passes=cfg.loop.times, name="step")) if looped else None,
        pass_vectors_name="loop",
        pass_input=PartSpec("stream_mix", dict(init_std=(2 * W) ** -0.5)) if looped else None,
        pass_input_name="loop.in",
        source=cfg,
    )


def fusion_rules(cfg: VodatarConfig) -> List[FusionRule]:
    """How checkpoint tensors combine into (or are renamed to) the model's tensors."""
    one = lambda target, source: FusionRule(target, [source], "same")  # noqa: E731  (a plain rename)
    rules = [one("embed_tokens.weight", "embed"), one("embed_tokens.norm.weight", "embed.norm"),
             one("head.weight", "head"), one("final.norm.weight", "final.norm")]
    if cfg.loop is not None:
        rules.append(one("loop.in.weight", "loop.in"))
    for i, l in enumerate(cfg.layers):
        p = f"l{i}"
        a = l.mixer
        if l.type == "attention":
            sizes = [a.heads * 2 * a.dim, a.kv_heads * 2 * a.dim, a.kv_heads * a.vdim]
            rules += [FusionRule(f"{p}.mix.qkv_proj.weight", [f"{p}.mix.{n}" for n in ("q", "k", "v")], "cat0", sizes),
                      FusionRule(f"{p}.mix.conv.weight", [f"{p}.mix.{n}.conv" for n in ("q", "k", "v")], "cat0", sizes),
                      one(f"{p}.mix.o_proj.weight", f"{p}.mix.o")]
        else:
            rules += [one(f"{p}.mix.in_proj.weight", f"{p}.mix.dkv"), one(f"{p}.mix.kv_norm.weight", f"{p}.mix.dkv.norm"),
                      one(f"{p}.mix.q_up.weight", f"{p}.mix.q"), one(f"{p}.mix.k_up.weight", f"{p}.mix.uk"),
                      one(f"{p}.mix.v_up.weight", f"{p}.mix.uv"), one(f"{p}.mix.o_proj.weight", f"{p}.mix.o")]
        f = l.mlp
        if f is None:
            continue
        rules += [FusionRule(f"{p}.mlp.experts.gate_up_proj",
                             [f"{p}.mlp.e{e}.{w}" for e in range(f.experts) for w in ("gate", "up")], "stack_pairs"),
                  FusionRule(f"{p}.mlp.experts.down_proj", [f"{p}.mlp.e{e}.down" for e in range(f.experts)], "stack"),
                  one(f"{p}.mlp.gate.weight", f"{p}.mlp.router"),
                  one(f"{p}.mlp.e_score_correction_bias", f"{p}.mlp.correction")]
        if f.shared_ff:
            rules += [FusionRule(f"{p}.mlp.shared_experts.gate_up_proj.weight",
                                 [f"{p}.mlp.shared.gate", f"{p}.mlp.shared.up"], "cat0"),
                      one(f"{p}.mlp.shared_experts.down_proj.weight", f"{p}.mlp.shared.down"),
                      one(f"{p}.mlp.shared_gate.weight", f"{p}.mlp.shared.sg")]
    return rules


def parse(raw: Mapping[str, Any], num_layers: Optional[int] = None) -> VodatarConfig:
    return VodatarConfig.from_dict(raw, num_layers=num_layers)


ARCH = Architecture(names=ARCHITECTURES, parse_config=parse, build_spec=build_spec, fusion_rules=fusion_rules)
register_architecture(ARCH)
