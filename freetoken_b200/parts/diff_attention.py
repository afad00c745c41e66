"""Differential attention: two softmax maps a head over the same values, the second taken off the first.

Per token, with ``H`` heads on ``G`` key/value heads, maps of ``dim`` and values of ``v_head_dim``::

    q, k, v = conv(W_q h), conv(W_k h), conv(W_v h)      a causal convolution over time on every channel
    q_h = [q_h1 | q_h2],  k_g = [k_g1 | k_g2]            each map turned by its token's position
    a_m = softmax_j(cap(q_hm(i) . k_gm(j) scale)) v_g(j)  cap(s) = softcap tanh(s / softcap), where there is a soft cap
    lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff      one number for the layer
    o_h = unit(a_1 - lambda a_2) (1 - diff)              unit: divided by the root mean square over the head

The cache holds ``[k_g1 | k_g2]`` and ``v_g`` as rows of one length, and query (head, map) is a row of that length that is
zero outside its map's place, so the two maps of a head are two more query heads on the same cached rows and the attention
kernels are the framework's own (:func:`ops.paged_attention`): every key and value is read once for both maps.  With
``2 dim = v_head_dim`` nothing is padded.  Convolution, rotation and the scatter into the pages are one kernel, and so is
the difference with its norm.  Rotation, scores, softmax and norm are 32-bit.

The mixer keeps pages (keys and values) and, with more than one tap, a state (the projections' last ``taps - 1`` rows).
The reference has no such layer.
"""

from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from ..config.spec import PagedKVNeed, ParamSpec, PartSpec, StateNeed
from ..engine.attention_plan import DEAL_MOST_PIECES
from ..errors import ConfigError
from ..kernels import ops
from .attention import TC_PAIR_MIN_TOKENS_LONG, attention_kernel_form
from .base import MIXERS, BuildEnv, Mixer, StepState
from .rope import shared_position

MAPS = 2


@MIXERS.register("differential_attention")
class DifferentialAttention(Mixer):
    """params: ``hidden``, ``n_heads``, ``n_kv_heads``, ``head_dim`` (of one map), ``v_head_dim``, ``taps`` (of the
    convolution; 1 still weighs every channel), ``position`` (PartSpec of an interleaved rotary encoding, or none),
    ``scale``, ``softcap`` (None or positive), ``diff`` (the constant part of lambda), ``eps``, ``init_std``."""

    graph_safe = False  # the convolution's state moves on with every run of a step
    graph_recordable = True

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        g = lambda k: int(spec[k])  # noqa: E731
        self.hidden, self.n_heads, self.n_kv_heads = g("hidden"), g("n_heads"), g("n_kv_heads")
        self.dim, self.v_dim, self.taps = g("head_dim"), g("v_head_dim"), int(spec.get("taps", 1))
        if min(self.hidden, self.n_heads, self.n_kv_heads, self.dim, self.v_dim) < 1 or self.n_heads % self.n_kv_heads:
            raise ConfigError("differential_attention: sizes must be positive, n_heads a multiple of n_kv_heads")
        if not 1 <= self.taps <= 16:
            raise ConfigError(f"differential_attention: {self.taps} taps (1 to 16 taken)")
        self.key_dim = MAPS * self.dim
        self.pad_dim = -(-max(self.key_dim, self.v_dim) // 16) * 16
        if self.pad_dim > 256:
            raise ConfigError(f"differential_attention: two maps of {self.dim} and values of {self.v_dim} exceed 256, the "
                              "attention kernels' largest head")
        self.scale = float(spec.get("scale") or self.dim ** -0.5)
        self.softcap: Optional[float] = None if spec.get("softcap") is None else float(spec["softcap"])
        if self.softcap is not None and not self.softcap > 0:
            raise ConfigError("differential_attention: a soft cap must be positive")
        self.diff = float(spec["diff"])
        self.eps = float(spec.get("eps", 1e-6))
        self.position = shared_position(spec.get("position") or PartSpec("none"), env)
        self.n_rot = int(getattr(self.position, "rotary_dim", 0))
        self.interleaved = bool(getattr(self.position, "interleaved", False))
        if self.n_rot > self.dim or (self.n_rot and not self.interleaved):
            raise ConfigError("differential_attention: turns pairs of neighbours within a map")
        self.q_rows = self.n_heads * self.key_dim
        self.k_rows = self.n_kv_heads * self.key_dim
        self.v_rows = self.n_kv_heads * self.v_dim
        self.rows = self.q_rows + self.k_rows + self.v_rows
        self.q_heads = self.n_heads * MAPS  # rows a token brings to the attention kernels
        self.group = self.q_heads // self.n_kv_heads
        most = 16 if env.dtype != torch.bfloat16 else 64  # query rows on one KV head that a tile takes
        self.kv_split = next(s for s in range(1, self.group + 1) if self.group % s == 0 and self.group // s <= most)
        self.plan_group = self.group // self.kv_split
        self.plan_kv_heads = self.n_kv_heads * self.kv_split
        self._lambda: Optional[torch.Tensor] = None

    # ------------------------------------------------------------------ tensors
    def param_specs(self) -> Dict[str, ParamSpec]:
        std = self.spec.get("init_std")
        s_in, s_out = (float(std[0]), float(std[1])) if std else (0.02, 0.02)
        f32 = dict(dtype="float32", store="bfloat16")
        out = {
            "qkv_proj.weight": ParamSpec((self.rows, self.hidden), init=("normal", 0.0, s_in)),
            "conv.weight": ParamSpec((self.rows, self.taps), init=("normal", 0.5 if std else 1.0, 0.3 if std else 0.02), **f32),
            "o_proj.weight": ParamSpec((self.hidden, self.n_heads * self.v_dim), init=("normal", 0.0, s_out)),
        }
        for n in ("lq1", "lk1", "lq2", "lk2"):
            out[n] = ParamSpec((self.dim,), init=("normal", 0.0, 0.1), **f32)
        return out

    def bind(self, tensors) -> None:
        super().bind(tensors)
        p = self.params
        self._lambda = (torch.exp((p["lq1"] * p["lk1"]).sum()) - torch.exp((p["lq2"] * p["lk2"]).sum()) + self.diff).reshape(1)

    def cache_need(self):
        pages = PagedKVNeed((("k", self.n_kv_heads, self.pad_dim), ("v", self.n_kv_heads, self.pad_dim)), None)
        state = StateNeed((("conv", (self.taps - 1, self.rows), "float32"),)) if self.taps > 1 else None
        return (pages, state)

    def workspace_bytes(self, n_tokens: int) -> int:
        item = 4 if self.env.dtype == torch.float32 else 2
        rows = n_tokens * (self.rows + 2 * self.q_heads * self.pad_dim + self.n_heads * self.v_dim + self.hidden) * item
        return rows + DEAL_MOST_PIECES * 148 * 256 * (self.pad_dim + 2) * 4

    # ------------------------------------------------------------------ step
    def kernel_form(self, decode_only: bool, n_tokens: int = 0, page_size: int = 0, longest_span: int = 0):
        sized = self.kv_split == 1
        return attention_kernel_form(self.env.dtype, decode_only, self.plan_group, n_tokens, self.pad_dim if sized else 0,
                                     page_size, None, longest_span)

    def plan_key(self, decode_only: bool = False, n_tokens: int = 0, page_size: int = 0, longest_span: int = 0):
        rows, few = self.kernel_form(decode_only, n_tokens, page_size, longest_span)
        return ("attention", self.plan_group, rows, None, self.plan_kv_heads, self.pad_dim, few)

    def prepare(self, builder) -> None:
        n_tokens = sum(q for q, _ in builder.seg_lens)
        page_size = builder.engine.config.page_size if builder.engine is not None else 0
        rows, few = self.kernel_form(builder.decode_only, n_tokens, page_size, builder.longest_span())
        if rows >= 128 and not few and not builder.decode_only and n_tokens >= TC_PAIR_MIN_TOKENS_LONG \
                and hasattr(builder, "cheaper_attention_rows"):
            # one or two query tiles a piece: whichever work list the kernel is estimated to get through sooner
            rows = builder.cheaper_attention_rows(self.plan_group, None, self.plan_kv_heads, self.pad_dim)
        self._step_plan = builder.attention_plan(self.plan_group, rows, None, self.plan_kv_heads, self.pad_dim, few)

    def forward(self, h: torch.Tensor, step: StepState, cache: Any, writes_cache: bool) -> torch.Tensor:
        if not writes_cache:
            raise ConfigError("differential_attention: the layer owns its cache")
        pages, state = cache
        T = h.shape[0]
        ws, dt, cap = self.env.workspace, self.env.dtype, self.env.max_step_tokens
        H, P = self.q_heads, self.pad_dim
        proj = ws.get("diff.qkv", (T, self.rows), dt, (cap, self.rows))
        ops.linear(h, self.params["qkv_proj.weight"], proj)
        q = ws.get("diff.q", (T, H, P), dt, (cap, H, P))
        ops.conv_rope_store(proj, self.params["conv.weight"], state.tensors["conv"] if state is not None else None,
                            step.state_slots, step.seg_info, len(step.segments), self.n_heads, self.n_kv_heads, MAPS,
                            self.dim, self.v_dim, self.n_rot, self.interleaved, step.positions, self.position.table(),
                            q, pages.slabs["k"], pages.slabs["v"], pages.slot_map)
        plan = step.attention_plans[self._step_plan]
        o = ws.get("diff.o", (T, H, P), dt, (cap, H, P))
        ops.paged_attention(q, pages.slabs["k"], pages.slabs["v"], pages.block_table, step.seg_info, len(step.segments),
                            plan.items_dev, plan.n_items, plan.part_o, plan.part_ml, o, self._step_plan[2], self.scale, None,
                            few_rows=self._step_plan[6], kv_split=self.kv_split, softcap=self.softcap)
        d = ws.get("diff.heads", (T, self.n_heads, self.v_dim), dt, (cap, self.n_heads, self.v_dim))
        ops.diff_heads(o, self._lambda, self.eps, 1.0 - self.diff, d)
        out = ws.get("diff.out", (T, self.hidden), dt, (cap, self.hidden))
        ops.linear(d.view(T, self.n_heads * self.v_dim), self.params["o_proj.weight"], out)
        return out
