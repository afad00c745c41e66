"""Plain, slow Gizulorn: whole sequences, no cache, no batching, one function per mechanism.

Gizulorn is a pre-norm decoder.  A layer's mixer is either two mixers side by side on one input (windowed attention whose
first tokens stay visible, with a learned sink in the softmax; and a gated delta rule with a decay per key channel), whose
results are added with constant factors, or retention (linear attention with a fixed decay per head).  Feed-forward: a dense
gated layer, a mixture of experts in groups of which only the best few may be chosen from, with a gated shared expert, or
none.

The file shares no code with ``freetoken_b200``: it parses config.json and reads the safetensors file itself.
Everything is computed in the working dtype (float64 by default).
"""

from __future__ import annotations

import json
import math
import os
import struct
from typing import Dict, List, Optional, Sequence

import torch

UNIT_EPS = 1e-6  # inside the root that makes the delta rule's queries and keys unit vectors


# --------------------------------------------------------------------------- mechanisms
def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x [T, C]``, ``w [C, taps]``: the last tap meets the token itself, the one before it the token before, ..."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for back in range(min(taps, T)):
        out[back:] = out[back:] + w[:, taps - 1 - back] * x[: T - back]
    return out


def frequencies(rot: dict) -> List[float]:
    """One angular frequency per pair; with ``scaling`` the slow ones are divided by ``factor``, judged by how often a pair's
    wavelength fits into the original length."""
    dims, base, sc = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        if sc:
            original, low, high, factor = (float(sc[k]) for k in ("original", "low", "high", "factor"))
            length = 2.0 * math.pi / f
            if length > original / low:
                f = f / factor
            elif length >= original / high:
                share = (original / length - low) / (high - low)
                f = (1.0 - share) * f / factor + share * f
        out.append(f)
    return out


def rotate_neighbours(x: torch.Tensor, freqs: Sequence[float]) -> torch.Tensor:
    """``x [T, heads, dim]``: columns ``2i`` and ``2i + 1`` turn together; the columns behind the pairs stay."""
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=x.dtype)[:, None]
    for i, f in enumerate(freqs):
        c, s = torch.cos(p * f), torch.sin(p * f)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def rotate_halves(x: torch.Tensor, freqs: Sequence[float]) -> torch.Tensor:
    """The same with columns ``i`` and ``i + len(freqs)`` as a pair."""
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=x.dtype)[:, None]
    n = len(freqs)
    for i, f in enumerate(freqs):
        c, s = torch.cos(p * f), torch.sin(p * f)
        u, v = x[..., i], x[..., i + n]
        out[..., i], out[..., i + n] = u * c - v * s, v * c + u * s
    return out


def visible(T: int, size: Optional[int], keep_first: int) -> torch.Tensor:
    """``[query, key]``: the past, as far as it is in the window or among the kept first tokens."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = (i - j < size) if size is not None else torch.ones(T, T, dtype=torch.bool)
    return (j <= i) & (near | (j < keep_first))


def softmax_with_sink(s: torch.Tensor, sink: torch.Tensor) -> torch.Tensor:
    """Rows of scores; the sink takes its share of the weights and has no column in the result."""
    m = torch.maximum(s.amax(-1, keepdim=True), sink)
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def sink_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, D), (h @ w["k"].T).view(T, G, D), (h @ w["v"].T).view(T, G, Dv)
    if m.get("rot"):
        f = frequencies(m["rot"])
        q, k = rotate_neighbours(q, f), rotate_neighbours(k, f)
    mask = m.get("mask") or {}
    ok = visible(T, mask.get("size"), int(mask.get("keep_first", 0)))
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = ((q[:, a] @ k[:, g].T) * m["scale"]).masked_fill(~ok, float("-inf"))
        heads.append(softmax_with_sink(s, w["sink"][a]) @ v[:, g])
    return torch.cat(heads, -1) @ w["o"].T


def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, beta: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
    """One head: ``q, k, g [T, D]``, ``v [T, Dv]``, ``beta [T]``; the state's rows belong to key channels."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype)
    out = torch.zeros_like(v)
    for t in range(v.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


def channel_delta(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[n].T, w[n + ".conv"])) for n in ("q", "k", "v"))
    q, k, v = q.view(T, G, D), k.view(T, G, D), v.view(T, H, Dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + UNIT_EPS) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + UNIT_EPS)
    beta = torch.sigmoid(h @ w["b"].T)
    rate = torch.nn.functional.softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(T, H, D)
    decay = torch.exp(-torch.exp(w["A_log"])[:, None] * rate)
    gate = torch.sigmoid((h @ w["g1"].T) @ w["g2"].T)
    heads = [over_rms(delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], beta[:, a], decay[:, a]), eps) * w["norm"]
             for a in range(H)]
    return (torch.cat(heads, -1) * gate) @ w["o"].T


def side_by_side(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    def under(p):
        return {n[len(p):]: t for n, t in w.items() if n.startswith(p)}

    return (float(m["left_scale"]) * sink_attention(h, under("left."), m["left"], eps)
            + float(m["right_scale"]) * channel_delta(h, under("right."), m["right"], eps))


def retention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w["q"].T).view(T, H, D), (h @ w["k"].T).view(T, H, D), (h @ w["v"].T).view(T, H, Dv)
    if m.get("rot"):
        f = frequencies(m["rot"])
        q, k = rotate_halves(q, f), rotate_halves(k, f)
    k = k * D ** -0.5
    heads = []
    for a in range(H):
        S = torch.zeros(D, Dv, dtype=h.dtype)
        o = torch.zeros(T, Dv, dtype=h.dtype)
        for t in range(T):
            S = float(m["decay"][a]) * S + torch.outer(k[t, a], v[t, a])
            o[t] = S.T @ q[t, a]
        heads.append(over_rms(o, eps))
    return (torch.cat(heads, -1) * silu(h @ w["g"].T)) @ w["o"].T


def gated_layer(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def choose_experts(s: torch.Tensor, top: int, groups: int, keep: int):
    """``s [T, experts]`` scores.  ``(chosen [T, top], gap [T])``; ``gap``: the smaller of the leads of the last kept group
    over the next one and of the last chosen expert over the next one that could have been."""
    T, E = s.shape
    best = s.view(T, groups, E // groups).amax(-1)
    order = torch.argsort(best, dim=-1, descending=True, stable=True)
    open_ = torch.zeros(T, groups, dtype=torch.bool).scatter(-1, order[:, :keep], True)
    can = s.masked_fill(~open_.repeat_interleave(E // groups, dim=-1), float("-inf"))
    rank = torch.argsort(can, dim=-1, descending=True, stable=True)
    gap = torch.full((T,), math.inf, dtype=s.dtype)
    if keep < groups:
        b = best.gather(-1, order)
        gap = torch.minimum(gap, b[:, keep - 1] - b[:, keep])
    if top < E:
        r = can.gather(-1, rank)
        gap = torch.minimum(gap, r[:, top - 1] - r[:, top])
    return rank[:, :top], gap


def mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, gaps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    s = torch.softmax(h @ w["router"].T, -1)
    chosen, gap = choose_experts(s, int(r["top"]), int(groups["count"]), int(groups["keep"]))
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in chosen[t].tolist():
            out[t] = out[t] + s[t, e] * gated_layer(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    if m.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * gated_layer(h, w["shared.gate"], w["shared.up"], w["shared.down"])
    return out


MIXERS = {"parallel": side_by_side, "retention": retention}


# --------------------------------------------------------------------------- files
def read_safetensors(path: str) -> Dict[str, torch.Tensor]:
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        meta = json.loads(f.read(n))
        data = f.read()
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "I32": torch.int32, "F16": torch.float16}
    out = {}
    for name, info in meta.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[lo:hi]), dtype=kinds[info["dtype"]]).view(info["shape"]).clone()
    return out


class PlainGizulorn:
    def __init__(self, folder: Optional[str] = None, raw: Optional[dict] = None,
                 weights: Optional[Dict[str, torch.Tensor]] = None, dtype: torch.dtype = torch.float64):
        if raw is None:
            with open(os.path.join(folder, "config.json")) as f:
                raw = json.load(f)
        if weights is None:
            weights = read_safetensors(os.path.join(folder, "model.safetensors"))
        self.raw = raw
        self.dtype = dtype
        self.w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in weights.items()}
        self.eps = float(raw["norm"]["eps"])
        self.vocab = int(raw["vocab"])

    def sub(self, prefix: str) -> Dict[str, torch.Tensor]:
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return over_rms(x, self.eps) * self.w[name]

    def forward(self, tokens: Sequence[int], layers_out: Optional[List[torch.Tensor]] = None,
                gaps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Logits ``[T, vocab]``; with ``layers_out`` the stream after every layer."""
        x = self.w["embed"][torch.tensor(list(tokens))]
        for i, layer in enumerate(self.raw["layers"]):
            p = f"l{i}."
            x = x + MIXERS[layer["type"]](self.norm(x, p + "norm1"), self.sub(p + "mix."), layer["mixer"], self.eps)
            f = layer.get("mlp")
            if f is not None:
                h, w = self.norm(x, p + "norm2"), self.sub(p + "mlp.")
                x = x + (gated_layer(h, w["gate"], w["up"], w["down"]) if f["kind"] == "dense" else mixture(h, w, f, gaps))
            if layers_out is not None:
                layers_out.append(x.clone())
        return self.norm(x, "final.norm") @ self.w["head"].T

    def logits(self, tokens: Sequence[int]) -> torch.Tensor:
        return self.forward(tokens).float()

    def layer_sums(self, tokens: Sequence[int]) -> List[torch.Tensor]:
        """The stream after every layer, float32."""
        out: List[torch.Tensor] = []
        self.forward(tokens, out)
        return [x.float() for x in out]

    def router_gaps(self, tokens: Sequence[int]) -> torch.Tensor:
        """Per token the smallest lead of a choice (group or expert) over the next one, over all layers."""
        gaps: List[torch.Tensor] = []
        self.forward(tokens, gaps=gaps)
        return torch.stack(gaps).min(0).values if gaps else torch.full((len(tokens),), math.inf, dtype=self.dtype)
