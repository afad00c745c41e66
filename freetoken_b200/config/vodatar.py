"""Typed Vodatar configuration, read from the design's own config.json keys.

A Vodatar file gives every size and every constant that can differ between models of the design:

* ``vocab``, ``width``, ``norm.eps``, ``norm.groups`` (equal parts of a row that are normed on their own),
  ``residual_mult`` (the factor on every sub-layer's normed result), ``canon.taps`` (of the convolutions in front of every
  sub-layer);
* ``loop`` (absent: every layer runs once): layers ``start .. stop - 1`` run ``times`` times in a row with the same weights;
* ``layers``: a list, one entry per layer, ``{"type", "mixer": {...}, "mlp": {...} | null}``.
  ``type: "attention"``: ``heads``, ``kv_heads``, ``dim`` (of one of a head's two maps), ``vdim``, ``conv`` (taps of the
  convolutions on q, k and v), ``scale``, ``softcap`` (absent: none), ``diff`` (the constant part of lambda), ``rot.dims``
  and ``rot.base``.
  ``type: "latent_attention"``: ``heads``, ``dim`` (unrotated query/key size per head), ``rot_dim`` (rotated size; the key's
  rotated part is shared by all heads), ``vdim``, ``kv_rank``, ``scale``, ``rot``.
  ``rot.scaling`` (either type; absent: none): ``factor``, ``original``, ``fast``, ``slow`` of YaRN.
  ``mlp.kind`` is ``"moe"``: ``expert.ff``, ``router.experts``, ``router.identity`` (experts that hand their input back,
  behind the others), ``router.top``, ``shared.ff`` (absent: no shared expert).

Anything missing or out of range becomes a :class:`ConfigError` naming the key.  The reference has no such
design; the reader follows the shape of its MiniMax-M3 reader (python/freetoken/models/minimax_m3/args.py:78-254).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from ..errors import ConfigError
from .pabavik import _get

ARCHITECTURES = ("Vodatar",)
MAX_POSITION = 1 << 20  # the design has no position limit of its own; tables are sized by the engine's longest sequence
MAX_TAPS = 16


@dataclass(frozen=True)
class VodatarRotation:
    dims: int
    base: float
    yarn: Optional[Tuple[float, float, float, float]] = None  # factor, original, fast, slow


@dataclass(frozen=True)
class VodatarAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    scale: float
    softcap: Optional[float]
    diff: float
    rot: Optional[VodatarRotation]


@dataclass(frozen=True)
class VodatarLatentAttention:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    rot: Optional[VodatarRotation]


@dataclass(frozen=True)
class VodatarMoe:
    ff: int
    experts: int
    identity: int
    top: int
    shared_ff: int


@dataclass(frozen=True)
class VodatarLayer:
    type: str  # "attention" | "latent_attention"
    mixer: Any
    mlp: Optional[VodatarMoe]


@dataclass(frozen=True)
class VodatarLoop:
    start: int
    stop: int
    times: int


def _positive(where: str, **values: float) -> None:
    for k, v in values.items():
        if not v > 0:
            raise ConfigError(f"config.json: '{where}{k}'={v} must be positive")


def _taps(where: str, key: str, v: int) -> int:
    if not 1 <= v <= MAX_TAPS:
        raise ConfigError(f"config.json: '{where}{key}'={v} must be in [1, {MAX_TAPS}]")
    return v


def _rotation(raw: Optional[Mapping[str, Any]], where: str, limit: int, default_dims: Optional[int]) -> Optional[VodatarRotation]:
    if not raw:
        return None
    dims = _get(raw, "dims", where, int) if default_dims is None or "dims" in raw else default_dims
    if dims == 0:
        return None
    base = float(_get(raw, "base", where, float))
    if dims < 0 or dims % 2 or dims > limit:
        raise ConfigError(f"config.json: '{where}dims'={dims} must be even and at most {limit}")
    _positive(where, base=base)
    s = raw.get("scaling")
    if s is None:
        return VodatarRotation(dims, base)
    w = where + "scaling."
    yarn = tuple(float(_get(s, k, w, float)) for k in ("factor", "original", "fast", "slow"))
    _positive(w, factor=yarn[0], original=yarn[1], fast=yarn[2], slow=yarn[3])
    if base == 1.0:
        raise ConfigError(f"config.json: '{where}base'=1 has no stretched frequencies")
    return VodatarRotation(dims, base, yarn)


@dataclass(frozen=True)
class VodatarConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    norm_groups: int
    residual_mult: float
    canon_taps: int
    loop: Optional[VodatarLoop]
    layers: Tuple[VodatarLayer, ...]
    torch_dtype: Optional[str] = None

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @staticmethod
    def from_dict(raw: Mapping[str, Any], num_layers: Optional[int] = None) -> "VodatarConfig":
        arch = raw.get("architecture") or (raw.get("architectures") or [None])[0]
        if arch not in ARCHITECTURES:
            raise ConfigError(f"config.json: architecture {arch!r} is not Vodatar")
        vocab = _get(raw, "vocab", "", int)
        width = _get(raw, "width", "", int)
        _positive("", vocab=vocab, width=width)
        norm = raw.get("norm") or {}
        groups = _get(norm, "groups", "norm.", int)
        if groups < 1 or width % groups:
            raise ConfigError(f"config.json: 'norm.groups'={groups} must divide 'width'={width}")
        taps = _taps("canon.", "taps", _get(raw.get("canon") or {}, "taps", "canon.", int))
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
            if typ == "attention":
                cap = m.get("softcap")
                dim = _get(m, "dim", wm, int)
                mixer = VodatarAttention(
                    heads=_get(m, "heads", wm, int), kv_heads=_get(m, "kv_heads", wm, int), dim=dim,
                    vdim=_get(m, "vdim", wm, int), taps=_taps(wm, "conv", _get(m, "conv", wm, int)),
                    scale=float(_get(m, "scale", wm, float)),
                    softcap=None if cap is None else float(_get(m, "softcap", wm, float)),
                    diff=float(_get(m, "diff", wm, float)), rot=_rotation(m.get("rot"), wm + "rot.", dim, None))
                _positive(wm, heads=mixer.heads, kv_heads=mixer.kv_heads, dim=mixer.dim, vdim=mixer.vdim, scale=mixer.scale)
                if mixer.softcap is not None:
                    _positive(wm, softcap=mixer.softcap)
                if mixer.heads % mixer.kv_heads:
                    raise ConfigError(f"config.json: '{wm}heads' must be a multiple of 'kv_heads'")
            elif typ == "latent_attention":
                rot_dim = _get(m, "rot_dim", wm, int)
                mixer = VodatarLatentAttention(
                    heads=_get(m, "heads", wm, int), dim=_get(m, "dim", wm, int), rot_dim=rot_dim,
                    vdim=_get(m, "vdim", wm, int), kv_rank=_get(m, "kv_rank", wm, int),
                    scale=float(_get(m, "scale", wm, float)), rot=_rotation(m.get("rot"), wm + "rot.", rot_dim, rot_dim))
                _positive(wm, heads=mixer.heads, dim=mixer.dim, vdim=mixer.vdim, kv_rank=mixer.kv_rank, scale=mixer.scale)
                if rot_dim < 0:
                    raise ConfigError(f"config.json: '{wm}rot_dim'={rot_dim} must not be negative")
            else:
                raise ConfigError(f"config.json: '{w}type' is {typ!r}; this design's mixers are: 'attention', "
                                  f"'latent_attention'")
            mlp = None
            rm = l.get("mlp")
            if rm is not None:
                wf = w + "mlp."
                kind = _get(rm, "kind", wf)
                if kind != "moe":
                    raise ConfigError(f"config.json: '{wf}kind' is {kind!r}; known: 'moe'")
                r = _get(rm, "router", wf)
                shared = rm.get("shared")
                mlp = VodatarMoe(
                    ff=_get(_get(rm, "expert", wf), "ff", wf + "expert.", int),
                    experts=_get(r, "experts", wf + "router.", int),
                    identity=_get(r, "identity", wf + "router.", int) if "identity" in r else 0,
                    top=_get(r, "top", wf + "router.", int),
                    shared_ff=_get(shared, "ff", wf + "shared.", int) if shared else 0)
                _positive(wf, ff=mlp.ff, experts=mlp.experts, top=mlp.top)
                if mlp.identity < 0 or mlp.top > mlp.experts + mlp.identity:
                    raise ConfigError(f"config.json: '{wf}router.top'={mlp.top} of {mlp.experts} + {mlp.identity} experts")
                if shared:
                    _positive(wf + "shared.", ff=mlp.shared_ff)
            layers.append(VodatarLayer(typ, mixer, mlp))
        loop = None
        rl = raw.get("loop")
        if rl:
            loop = VodatarLoop(*(_get(rl, k, "loop.", int) for k in ("start", "stop", "times")))
            n = len(layers)
            if num_layers is not None:  # (a cut model keeps what is left of the range)
                loop = VodatarLoop(min(loop.start, n - 1), min(loop.stop, n), loop.times)
            if not 0 <= loop.start < loop.stop <= n or loop.times < 1:
                raise ConfigError(f"config.json: 'loop' runs layers {loop.start} .. {loop.stop} - 1 {loop.times} times, the model "
                                  f"has {n} layers")
        return VodatarConfig(architecture=str(arch), vocab=vocab, width=width,
                             norm_eps=float(_get(norm, "eps", "norm.", float)), norm_groups=groups,
                             residual_mult=float(_get(raw, "residual_mult", "", float)), canon_taps=taps, loop=loop,
                             layers=tuple(layers), torch_dtype=raw.get("torch_dtype"))
