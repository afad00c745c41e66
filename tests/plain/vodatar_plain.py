"""Plain, slow Vodatar: whole sequences, no cache, no batching, one function per mechanism.

Vodatar is a decoder whose sub-layers are normed on both sides (RMS norms that take their mean over groups of
channels), read their normed input through a short causal convolution over time and write their result through a
gate computed from that input before the convolution.  A range of layers runs several times over with the same
weights; each pass starts by mixing the stream with the embedding output and adding a vector of the pass.  Mixers:
differential attention (two softmax maps over the same values, one subtracted from the other), whose projections
pass a short convolution before an interleaved rotation and whose scores are soft-capped; and latent attention with
rotation frequencies stretched for longer contexts.  Feed-forward: a mixture of experts, some of which hand their
input back, with a gated shared expert.

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


# --------------------------------------------------------------------------- mechanisms
def unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    """``x / sqrt(mean(x^2) + eps)`` over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def group_norm(x: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> torch.Tensor:
    """Each of ``groups`` equal consecutive parts of a row is divided by its own root mean square; then the weight."""
    parts = [unit(p, eps) for p in x.split(x.shape[-1] // groups, dim=-1)]
    return torch.cat(parts, -1) * w


def causal_conv(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x [T, C]``, ``w [C, taps]``: ``sum_j w[:, j] x_(t - taps + 1 + j)``, zeros before the start."""
    T, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for j in range(taps):
        back = taps - 1 - j  # how many places back this tap reads
        if back < T:
            out[back:] = out[back:] + w[:, j] * x[: T - back]
    return out


def plain_frequencies(dims: int, base: float) -> List[float]:
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def yarn_frequencies(dims: int, base: float, factor: float, original: float, fast: float, slow: float) -> List[float]:
    """Frequencies that turn at least ``fast`` times over the original context stay, those that turn at most
    ``slow`` times are divided by ``factor``, with a ramp over the index in between."""
    def index_of(turns: float) -> float:
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(index_of(fast)), 0)
    hi = min(math.ceil(index_of(slow)), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(dims, base)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out


def frequencies(rot: dict):
    """``(one frequency per pair, the factor on cosines and sines)`` of a config's ``rot``."""
    dims, base, s = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    if s is None:
        return plain_frequencies(dims, base), 1.0
    return (yarn_frequencies(dims, base, float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])),
            0.1 * math.log(float(s["factor"])) + 1.0)


def rotate_neighbours(x: torch.Tensor, freqs: Sequence[float], magnitude: float = 1.0) -> torch.Tensor:
    """``x [T, ..., dim]``: columns ``2i`` and ``2i + 1`` turn together by ``t freqs[i]``; the columns behind stay."""
    out = x.clone()
    p = torch.arange(x.shape[0], dtype=x.dtype).view([-1] + [1] * (x.dim() - 2))
    for i, f in enumerate(freqs):
        c, s = torch.cos(p * f) * magnitude, torch.sin(p * f) * magnitude
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def causal_softmax(s: torch.Tensor) -> torch.Tensor:
    T = s.shape[0]
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
    return torch.softmax(s, -1)


def differential_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(n):
        u = h @ w[n].T
        return causal_conv(u, w[n + ".conv"]) if n + ".conv" in w else u

    q = projected("q").view(T, H, 2, D)
    k = projected("k").view(T, G, 2, D)
    v = projected("v").view(T, G, Dv)
    rot = m.get("rot")
    if rot:
        freqs, mag = frequencies(rot)
        q, k = rotate_neighbours(q, freqs, mag), rotate_neighbours(k, freqs, mag)
    lam = torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + m["diff"]
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        maps = []
        for n in (0, 1):
            s = (q[:, a, n] @ k[:, g, n].T) * m["scale"]
            if m.get("softcap") is not None:
                s = m["softcap"] * torch.tanh(s / m["softcap"])
            maps.append(causal_softmax(s) @ v[:, g])
        out[:, a] = unit(maps[0] - lam * maps[1], eps) * (1.0 - m["diff"])
    return out.reshape(T, H * Dv) @ w["o"].T


def latent_attention(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, D, R, Dv, C = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    freqs, mag = frequencies(m["rot"])
    q = (h @ w["q"].T).view(T, H, D + R)
    q_flat, q_rot = q[..., :D], rotate_neighbours(q[..., D:], freqs, mag)
    kv = h @ w["dkv"].T
    c = unit(kv[:, :C], eps) * w["dkv.norm"]
    k_rot = rotate_neighbours(kv[:, C:], freqs, mag)  # [T, R], one for all heads
    k_flat = (c @ w["uk"].T).view(T, H, D)
    v = (c @ w["uv"].T).view(T, H, Dv)
    out = torch.zeros(T, H, Dv, dtype=h.dtype)
    for a in range(H):
        out[:, a] = causal_softmax((q_flat[:, a] @ k_flat[:, a].T + q_rot[:, a] @ k_rot.T) * m["scale"]) @ v[:, a]
    return out.reshape(T, H * Dv) @ w["o"].T


def gated_expert(h: torch.Tensor, gate: torch.Tensor, up: torch.Tensor, down: torch.Tensor) -> torch.Tensor:
    z = h @ gate.T
    return ((z * torch.sigmoid(z)) * (h @ up.T)) @ down.T


def choose_experts(h: torch.Tensor, router: torch.Tensor, correction: torch.Tensor, top: int):
    """``(chosen [T, top], weights [T, top], gap [T])``; ``gap``: by how much the last chosen one is ahead."""
    s = torch.softmax(h @ router.T, -1)
    choice = s + correction
    order = torch.argsort(choice, dim=-1, descending=True, stable=True)
    chosen = order[:, :top]
    weights = s.gather(-1, chosen)
    weights = weights / (weights.sum(-1, keepdim=True) + 1e-20)
    ranked = choice.gather(-1, order)
    gap = ranked[:, top - 1] - ranked[:, top] if top < ranked.shape[1] else torch.full_like(ranked[:, 0], math.inf)
    return chosen, weights, gap


def mixture(h: torch.Tensor, w: Dict[str, torch.Tensor], m: dict, gaps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
    r = m["router"]
    n_real = int(r["experts"])
    chosen, weights, gap = choose_experts(h, w["router"], w["correction"], int(r["top"]))
    if gaps is not None:
        gaps.append(gap)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, x in zip(chosen[t].tolist(), weights[t]):
            y = h[t] if e >= n_real else gated_expert(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
            out[t] = out[t] + x * y
    if m.get("shared"):
        y = gated_expert(h, w["shared.gate"], w["shared.up"], w["shared.down"])
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * y
    return out


MIXERS = {"attention": differential_attention, "latent_attention": latent_attention}


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


class PlainVodatar:
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
        self.groups = int(raw["norm"]["groups"])
        self.mult = float(raw["residual_mult"])
        self.vocab = int(raw["vocab"])

    def sub(self, prefix: str) -> Dict[str, torch.Tensor]:
        return {k[len(prefix):]: v for k, v in self.w.items() if k.startswith(prefix)}

    def norm(self, x: torch.Tensor, name: str) -> torch.Tensor:
        return group_norm(x, self.w[name], self.groups, self.eps)

    def passes(self) -> List[tuple]:
        """``(layer, number of the pass that starts right before it or None)`` in the order layers run."""
        n, loop = len(self.raw["layers"]), self.raw.get("loop")
        if not loop:
            return [(i, None) for i in range(n)]
        a, b = loop["start"], loop["stop"]
        out = [(i, None) for i in range(a)]
        for t in range(loop["times"]):
            out += [(i, t if i == a else None) for i in range(a, b)]
        return out + [(i, None) for i in range(b, n)]

    def sublayer(self, x: torch.Tensor, p: str, q: str, body) -> torch.Tensor:
        """``x + m norm_b(gate * body(h + conv(h)))`` with ``h = norm(x)``; ``q`` is "1" (mixer) or "2" (feed-forward)."""
        w = self.w
        h = self.norm(x, p + "norm" + q)
        y = body(h + causal_conv(h, w[p + "canon" + q]))
        y = y * torch.sigmoid(h @ w[p + "rg" + q].T + w[p + "rg" + q + ".b"])
        return x + self.mult * self.norm(y, p + "norm" + q + "b")

    def forward(self, tokens: Sequence[int], layers_out: Optional[List[torch.Tensor]] = None,
                gaps: Optional[List[torch.Tensor]] = None) -> torch.Tensor:
        """Logits ``[T, vocab]``; with ``layers_out`` the stream after every layer run."""
        w = self.w
        x = x0 = self.norm(w["embed"][torch.tensor(list(tokens))], "embed.norm")
        for i, start in self.passes():
            if start is not None:
                x = torch.cat([x, x0], -1) @ w["loop.in"].T + w["loop.step"][start]
            layer, p = self.raw["layers"][i], f"l{i}."
            mixer = MIXERS[layer["type"]]
            x = self.sublayer(x, p, "1", lambda u: mixer(u, self.sub(p + "mix."), layer["mixer"], self.eps))
            if layer.get("mlp") is not None:
                x = self.sublayer(x, p, "2", lambda u: mixture(u, self.sub(p + "mlp."), layer["mlp"], gaps))
            if layers_out is not None:
                layers_out.append(x.clone())
        return self.norm(x, "final.norm") @ w["head"].T

    def logits(self, tokens: Sequence[int]) -> torch.Tensor:
        return self.forward(tokens).float()

    def layer_sums(self, tokens: Sequence[int]) -> List[torch.Tensor]:
        """The stream after every layer run, float32."""
        out: List[torch.Tensor] = []
        self.forward(tokens, out)
        return [x.float() for x in out]

    def router_gaps(self, tokens: Sequence[int]) -> torch.Tensor:
        """Per token the smallest lead of a last chosen expert over the next one, over all layer runs."""
        gaps: List[torch.Tensor] = []
        self.forward(tokens, gaps=gaps)
        return torch.stack(gaps).min(0).values if gaps else torch.full((len(tokens),), math.inf, dtype=self.dtype)
