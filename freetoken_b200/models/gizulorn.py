"""Gizulorn: from its typed config to a model description, and its checkpoint names.

Layers are plain ``prenorm_residual`` blocks.  The mixer is ``side_by_side`` of ``gqa_attention`` (a sliding window that
keeps the first tokens, a learned sink per head, interleaved rotation with frequencies scaled in bands) and ``gated_delta``
(a decay per key channel and the output gate through low ranks), added with constant factors; or ``retention`` (a fixed
decay per head).  The feed-forward is ``gated_mlp``, ``moe`` (softmax scores as they are, experts in groups, a gated shared
expert) or none.

Checkpoint names: ``embed``, ``head``, ``final.norm`` and, per layer ``l<i>``: ``norm1``, ``norm2``; the pair
``mix.left.{q,k,v,sink,o}``, ``mix.right.{q,k,v}`` (each with ``.conv``), ``mix.right.{b,A_log,norm,a1,a2,dt_bias,g1,g2,o}``;
retention ``mix.{q,k,v,g,o}``; ``mlp.{gate,up,down}``, or ``mlp.e<j>.{gate,up,down}``, ``mlp.router``,
``mlp.shared.{gate,up,down,sg}``.  The projections of a mixer's input are concatenated into one matrix; gate/up pairs and
experts are stacked as for every other architecture here.  The reference has no such design.
"""

from __future__ import annotations

from dataclasses import replace
from typing import Any, List, Mapping, Optional, Tuple

from ..config.gizulorn import ARCHITECTURES, DEFAULT_RANK, MAX_POSITION, GizulornConfig, GizulornRotation
from ..config.spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry
from ..errors import ConfigError
from ..registry import Architecture, register_architecture
from ..weights.binder import FusionRule


def _position(rot: Optional[GizulornRotation], kind: str) -> PartSpec:
    if rot is None:
        return PartSpec("none")
    return PartSpec(kind, dict(rotary_dim=rot.dims, theta=rot.base, precise=True, band_scaling=rot.bands))


def build_spec(cfg: GizulornConfig) -> ModelSpec:
    W, eps = cfg.width, cfg.norm_eps
    # random models: spreads that keep every activation of order one, so that a fault anywhere shows in the logits
    w_in = W ** -0.5
    norm = PartSpec("rmsnorm", dict(size=W, eps=eps, gemma=False))
    block = PartSpec("prenorm_residual", dict(hidden=W, norm=norm, input_norm_name="norm1", post_norm_name="norm2"))
    layers: List[LayerSpec] = []
    for i, l in enumerate(cfg.layers):
        a = l.mixer
        if l.type == "parallel":
            le, ri = a.left, a.right
            left = PartSpec("gqa_attention", dict(
                hidden=W, n_heads=le.heads, n_kv_heads=le.kv_heads, head_dim=le.dim, v_head_dim=le.vdim, qk_norm=False, eps=eps,
                gemma=False, position=_position(le.rot, "rope_interleaved"), scale=le.scale, window=le.window,
                keep_first=le.keep_first, sink="learned", init_std=(w_in, (le.heads * le.vdim) ** -0.5)))
            right = PartSpec("gated_delta", dict(
                hidden=W, n_heads=ri.heads, n_kv_heads=ri.kv_heads, head_dim=ri.dim, v_head_dim=ri.vdim, taps=ri.taps, eps=eps,
                decay_rank=ri.decay_rank or DEFAULT_RANK, gate_rank=ri.gate_rank or DEFAULT_RANK, gate="sigmoid",
                init_std=(w_in, (ri.heads * ri.vdim) ** -0.5)))
            mixer = PartSpec("side_by_side", dict(hidden=W, branches=(("left", left), ("right", right)),
                                                  scales=(a.left_scale, a.right_scale)))
        else:
            mixer = PartSpec("retention", dict(
                hidden=W, n_heads=a.heads, head_dim=a.dim, v_head_dim=a.vdim, decay=a.decay, eps=eps,
                position=_position(a.rot, "rope_neox"), init_std=(w_in, (a.heads * a.vdim) ** -0.5)))
        f = l.mlp
        if f is None:
            ffn = PartSpec("none")
        elif f.kind == "dense":
            ffn = PartSpec("gated_mlp", dict(hidden=W, inter=f.ff, act="silu", init_std=(w_in, f.ff ** -0.5)))
        else:
            ffn = PartSpec("moe", dict(hidden=W, inter=f.ff, n_experts=f.experts, top_k=f.top, scoring="softmax_raw",
                                       groups=(f.groups, f.keep_groups), bias=False, scale=1.0, act="silu",
                                       shared_inter=f.shared_ff, shared_gate=bool(f.shared_ff), router_store="bfloat16",
                                       init_std=(w_in, f.ff ** -0.5)))
        layers.append(LayerSpec(name=f"l{i}", block=block, mixer=mixer, ffn=ffn, mixer_name="mix", ffn_name="mlp"))
    return ModelSpec(
        architecture=cfg.architecture, vocab_size=cfg.vocab, hidden_size=W, layers=tuple(layers),
        schedule=tuple(ScheduleEntry(i, None) for i in range(len(layers))),
        embedding=PartSpec("token_embedding", dict(vocab=cfg.vocab, hidden=W, init_std=1.0)),
        final_norm=norm,
        head=PartSpec("linear_head", dict(tied=False, init_std=w_in)),
        max_position=MAX_POSITION,
        embedding_name="embed_tokens", final_norm_name="final.norm", head_name="head",
        source=cfg,
    )


def fusion_rules(cfg: GizulornConfig) -> List[FusionRule]:
    """How checkpoint tensors combine into (or are renamed to) the model's tensors."""
    one = lambda target, source: FusionRule(target, [source], "same")  # noqa: E731  (a plain rename)
    rules = [one("embed_tokens.weight", "embed"), one("head.weight", "head"), one("final.norm.weight", "final.norm")]
    for i, l in enumerate(cfg.layers):
        p = f"l{i}"
        a = l.mixer
        rules.append(one(f"{p}.norm1.weight", f"{p}.norm1"))
        if l.type == "parallel":
            le, ri = a.left, a.right
            m = f"{p}.mix.left"
            rules += [FusionRule(f"{m}.qkv_proj.weight", [f"{m}.{n}" for n in ("q", "k", "v")], "cat0",
                                 [le.heads * le.dim, le.kv_heads * le.dim, le.kv_heads * le.vdim]),
                      one(f"{m}.o_proj.weight", f"{m}.o")]
            m = f"{p}.mix.right"
            qkv = [ri.kv_heads * ri.dim, ri.kv_heads * ri.dim, ri.heads * ri.vdim]
            rules += [FusionRule(f"{m}.in_proj.weight", [f"{m}.{n}" for n in ("q", "k", "v", "g1", "b", "a1")], "cat0",
                                 qkv + [ri.gate_rank or DEFAULT_RANK, ri.heads, ri.decay_rank or DEFAULT_RANK]),
                      FusionRule(f"{m}.conv.weight", [f"{m}.{n}.conv" for n in ("q", "k", "v")], "cat0", qkv),
                      one(f"{m}.decay_proj.weight", f"{m}.a2"), one(f"{m}.gate_proj.weight", f"{m}.g2"),
                      one(f"{m}.norm.weight", f"{m}.norm"), one(f"{m}.o_proj.weight", f"{m}.o")]
        else:
            m = f"{p}.mix"
            rules += [FusionRule(f"{m}.in_proj.weight", [f"{m}.{n}" for n in ("q", "k", "v", "g")], "cat0",
                                 [a.heads * a.dim, a.heads * a.dim, a.heads * a.vdim, a.heads * a.vdim]),
                      one(f"{m}.o_proj.weight", f"{m}.o")]
        f = l.mlp
        if f is None:
            continue
        rules.append(one(f"{p}.norm2.weight", f"{p}.norm2"))
        m = f"{p}.mlp"
        if f.kind == "dense":
            rules += [FusionRule(f"{m}.gate_up_proj.weight", [f"{m}.gate", f"{m}.up"], "cat0"),
                      one(f"{m}.down_proj.weight", f"{m}.down")]
            continue
        rules += [FusionRule(f"{m}.experts.gate_up_proj", [f"{m}.e{e}.{w}" for e in range(f.experts) for w in ("gate", "up")],
                             "stack_pairs"),
                  FusionRule(f"{m}.experts.down_proj", [f"{m}.e{e}.down" for e in range(f.experts)], "stack"),
                  one(f"{m}.gate.weight", f"{m}.router")]
        if f.shared_ff:
            rules += [FusionRule(f"{m}.shared_experts.gate_up_proj.weight", [f"{m}.shared.gate", f"{m}.shared.up"], "cat0"),
                      one(f"{m}.shared_experts.down_proj.weight", f"{m}.shared.down"),
                      one(f"{m}.shared_gate.weight", f"{m}.shared.sg")]
    return rules


def parse(raw: Mapping[str, Any], num_layers: Optional[int] = None) -> GizulornConfig:
    return GizulornConfig.from_dict(raw, num_layers=num_layers)


def sizes_from_weights(cfg: GizulornConfig, shapes: Mapping[str, Tuple[int, ...]]) -> GizulornConfig:
    """The widths of the delta rule's low-rank projections are the first sizes of ``l<i>.mix.right.a1`` and ``.g1``."""
    layers = list(cfg.layers)
    for i, l in enumerate(layers):
        if l.type != "parallel":
            continue
        found = {}
        for name, field in (("a1", "decay_rank"), ("g1", "gate_rank")):
            shape = shapes.get(f"l{i}.mix.right.{name}")
            if shape is None:
                continue
            if len(shape) != 2 or shape[0] < 1 or shape[1] != cfg.width:
                raise ConfigError(f"l{i}.mix.right.{name} has shape {list(shape)}: [rank >= 1, {cfg.width}] expected")
            found[field] = int(shape[0])
        layers[i] = replace(l, mixer=replace(l.mixer, right=replace(l.mixer.right, **found)))
    return replace(cfg, layers=tuple(layers))


ARCH = Architecture(names=ARCHITECTURES, parse_config=parse, build_spec=build_spec, fusion_rules=fusion_rules,
                    sizes_from_weights=sizes_from_weights)
register_architecture(ARCH)
