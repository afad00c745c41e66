"""Typed Gizulorn configuration, read from the design's own config.json keys.

A Gizulorn file gives every size and every constant that can differ between models of the design:

* ``vocab``, ``width``, ``norm.eps``;
* ``layers``: a list, one entry per layer, ``{"type", "mixer": {...}, "mlp": {...} | null}``.
  ``type: "parallel"``: two mixers on one input, added as ``left_scale * left + right_scale * right``.
  ``left`` (windowed attention): ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (a token sees itself and the
  ``size - 1`` before it) and ``mask.keep_first`` (first tokens that stay visible), ``rot`` (neighbours turn together).
  ``right`` (gated delta rule, a decay per key channel): ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv`` (taps); the widths of
  its two low-rank projections are tensor shapes and come from the weight file's header (a config written for random weights
  may say ``decay_rank`` and ``gate_rank``).
  ``type: "retention"``: ``heads``, ``dim``, ``vdim``, ``decay`` (a number per head), ``rot`` (halves turn together).
  ``rot`` (absent: no rotation): ``dims`` (leading dimensions of a head that turn), ``base`` and, optionally, ``scaling``:
  ``factor``, ``low``, ``high``, ``original``.
  ``mlp.kind`` is ``"dense"`` (``ff``) or ``"moe"``: ``expert.ff``, ``router.experts``, ``router.top``, ``router.groups.count`` and
  ``.keep`` (absent: one group), ``shared.ff`` (absent: no shared expert).

Anything missing or out of range becomes a :class:`ConfigError` naming the key.  The reference has no such
design; the reader follows the shape of its MiniMax-M3 reader (python/freetoken/models/minimax_m3/args.py:78-254).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ConfigError
from .pabavik import _get
from .vodatar import _positive, _taps

ARCHITECTURES = ("Gizulorn",)
MAX_POSITION = 1 << 20  # the design has no position limit of its own; tables are sized by the engine's longest sequence
DEFAULT_RANK = 16  # of a low-rank projection when neither a weight file nor the config says (random models)


@dataclass(frozen=True)
class GizulornRotation:
    dims: int
    base: float
    bands: Optional[Tuple[float, float, float, float]] = None  # factor, low, high, original


@dataclass(frozen=True)
class GizulornAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]
    keep_first: int
    rot: Optional[GizulornRotation]


@dataclass(frozen=True)
class GizulornDelta:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay_rank: int  # 0: not known yet
    gate_rank: int


@dataclass(frozen=True)
class GizulornParallel:
    left: GizulornAttention
    right: GizulornDelta
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class GizulornRetention:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: Optional[GizulornRotation]


@dataclass(frozen=True)
class GizulornMlp:
    kind: str  # "dense" | "moe"
    ff: int
    experts: int = 0
    top: int = 0
    groups: int = 1
    keep_groups: int = 1
    shared_ff: int = 0  # 0: no shared expert


@dataclass(frozen=True)
class GizulornLayer:
    type: str  # "parallel" | "retention"
    mixer: Any
    mlp: Optional[GizulornMlp]


def _rotation(raw: Optional[Mapping[str, Any]], where: str, limit: int) -> Optional[GizulornRotation]:
    if not raw:
        return None
    dims = _get(raw, "dims", where, int)
    if dims == 0:
        return None
    if dims < 0 or dims % 2 or dims > limit:
        raise ConfigError(f"config.json: '{where}dims'={dims} must be even and at most {limit}")
    base = float(_get(raw, "base", where, float))
    _positive(where, base=base)
    s = raw.get("scaling")
    if s is None:
        return GizulornRotation(dims, base)
    w = where + "scaling."
    bands = tuple(float(_get(s, k, w, float)) for k in ("factor", "low", "high", "original"))
    _positive(w, factor=bands[0], low=bands[1], high=bands[2], original=bands[3])
    return GizulornRotation(dims, base, bands)


def _attention(m: Mapping[str, Any], wm: str) -> GizulornAttention:
    dim = _get(m, "dim", wm, int)
    mask = m.get("mask") or {}
    window = mask.get("size")
    if window is not None:
        window = _get(mask, "size", wm + "mask.", int)
        _positive(wm + "mask.", size=window)
    keep = _get(mask, "keep_first", wm + "mask.", int) if "keep_first" in mask else 0
    if keep < 0:
        raise ConfigError(f"config.json: '{wm}mask.keep_first'={keep} must not be negative")
    a = GizulornAttention(heads=_get(m, "heads", wm, int), kv_heads=_get(m, "kv_heads", wm, int), dim=dim,
                          vdim=_get(m, "vdim", wm, int), scale=float(_get(m, "scale", wm, float)), window=window,
                          keep_first=keep if window is not None else 0, rot=_rotation(m.get("rot"), wm + "rot.", dim))
    _positive(wm, heads=a.heads, kv_heads=a.kv_heads, dim=dim, vdim=a.vdim, scale=a.scale)
    if a.heads % a.kv_heads:
        raise ConfigError(f"config.json: '{wm}heads' must be a multiple of 'kv_heads'")
    return a


def _delta(m: Mapping[str, Any], wm: str) -> GizulornDelta:
    ranks = [_get(m, k, wm, int) if k in m else 0 for k in ("decay_rank", "gate_rank")]
    d = GizulornDelta(heads=_get(m, "heads", wm, int), kv_heads=_get(m, "kv_heads", wm, int), dim=_get(m, "dim", wm, int),
                      vdim=_get(m, "vdim", wm, int), taps=_taps(wm, "conv", _get(m, "conv", wm, int)),
                      decay_rank=ranks[0], gate_rank=ranks[1])
    _positive(wm, heads=d.heads, kv_heads=d.kv_heads, dim=d.dim, vdim=d.vdim)
    if d.heads % d.kv_heads:
        raise ConfigError(f"config.json: '{wm}heads' must be a multiple of 'kv_heads'")
    if min(ranks) < 0:
        raise ConfigError(f"config.json: '{wm}decay_rank' and 'gate_rank' must not be negative")
    return d


def _mlp(rm: Mapping[str, Any], wf: str) -> GizulornMlp:
    kind = _get(rm, "kind", wf)
    if kind == "dense":
        mlp = GizulornMlp("dense", ff=_get(rm, "ff", wf, int))
        _positive(wf, ff=mlp.ff)
        return mlp
    if kind != "moe":
        raise ConfigError(f"config.json: '{wf}kind' is {kind!r}; known: 'dense', 'moe'")
    r = _get(rm, "router", wf)
    wr = wf + "router."
    groups, shared = r.get("groups"), rm.get("shared")
    mlp = GizulornMlp(
        "moe", ff=_get(_get(rm, "expert", wf), "ff", wf + "expert.", int), experts=_get(r, "experts", wr, int),
        top=_get(r, "top", wr, int), groups=_get(groups, "count", wr + "groups.", int) if groups else 1,
        keep_groups=_get(groups, "keep", wr + "groups.", int) if groups else 1,
        shared_ff=_get(shared, "ff", wf + "shared.", int) if shared else 0)
    _positive(wf, ff=mlp.ff, experts=mlp.experts, top=mlp.top)
    if shared:
        _positive(wf + "shared.", ff=mlp.shared_ff)
    if not 1 <= mlp.keep_groups <= mlp.groups or mlp.experts % mlp.groups:
        raise ConfigError(f"config.json: '{wr}groups': the best {mlp.keep_groups} of {mlp.groups} equal groups of {mlp.experts} experts")
    if mlp.top > mlp.experts // mlp.groups * mlp.keep_groups:
        raise ConfigError(f"config.json: '{wr}top'={mlp.top} exceeds the {mlp.experts // mlp.groups * mlp.keep_groups} experts that can "
                          f"be chosen")
    return mlp


@dataclass(frozen=True)
class GizulornConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: Tuple[GizulornLayer, ...]
    torch_dtype: Optional[str] = None

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @staticmethod
    def from_dict(raw: Mapping[str, Any], num_layers: Optional[int] = None) -> "GizulornConfig":
        arch = raw.get("architecture") or (raw.get("architectures") or [None])[0]
        if arch not in ARCHITECTURES:
            raise ConfigError(f"config.json: architecture {arch!r} is not Gizulorn")
        vocab, width = _get(raw, "vocab", "", int), _get(raw, "width", "", int)
        _positive("", vocab=vocab, width=width)
        raw_layers = _get(raw, "layers", "")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        if num_layers is not None:
            raw_layers = raw_layers[:max(1, num_layers)]
        layers = []
        for i, l in enumerate(raw_layers):
            w = f"layers[{i}]."
            typ = _get(l, "type", w)
            m = _get(l, "mixer", w)
            wm = w + "mixer."
            if typ == "parallel":
                mixer = GizulornParallel(
                    left=_attention(_get(m, "left", wm), wm + "left."), right=_delta(_get(m, "right", wm), wm + "right."),
                    left_scale=float(_get(m, "left_scale", wm, float)), right_scale=float(_get(m, "right_scale", wm, float)))
            elif typ == "retention":
                dim = _get(m, "dim", wm, int)
                decay = _get(m, "decay", wm)
                if not isinstance(decay, list) or any(isinstance(x, bool) or not isinstance(x, (int, float)) for x in decay):
                    raise ConfigError(f"config.json: '{wm}decay' must be a list of numbers")
                mixer = GizulornRetention(heads=_get(m, "heads", wm, int), dim=dim, vdim=_get(m, "vdim", wm, int),
                                          decay=tuple(float(x) for x in decay), rot=_rotation(m.get("rot"), wm + "rot.", dim))
                _positive(wm, heads=mixer.heads, dim=dim, vdim=mixer.vdim)
                if len(mixer.decay) != mixer.heads:
                    raise ConfigError(f"config.json: '{wm}decay' holds {len(mixer.decay)} numbers for {mixer.heads} heads")
            else:
                raise ConfigError(f"config.json: '{w}type' is {typ!r}; this design's mixers are: 'parallel', 'retention'")
            rm = l.get("mlp")
            layers.append(GizulornLayer(typ, mixer, None if rm is None else _mlp(rm, w + "mlp.")))
        return GizulornConfig(architecture=str(arch), vocab=vocab, width=width,
                              norm_eps=float(_get(raw.get("norm") or {}, "eps", "norm.", float)), layers=tuple(layers),
                              torch_dtype=raw.get("torch_dtype"))
