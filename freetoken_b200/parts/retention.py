"""Retention: linear attention with a fixed decay per head.

One projection of the input gives ``[q | k | v | g]``: queries and keys ``[n_heads, head_dim]``, values and an output gate
``[n_heads, v_head_dim]``.  Queries and keys are rotated by their position; per token and head::

    S_t = a_h S_(t-1) + k_t v_t^T          o_t = S_t^T q_t head_dim^-1/2

without softmax or denominator.  Each head's ``o_t`` is divided by its root mean square (no weight), multiplied element by
element by ``silu`` of the gate and projected.

The recurrence is :func:`ops.gla_scan` with one row of decays for every token; the rotation is taken in 32 bits while that
kernel reads the projection's rows, so that what enters the recurrence is not rounded.  State, decays and outputs are
32-bit, norm and gate :func:`ops.gated_heads`.  The state (``[n_heads, head_dim, v_head_dim]``) lives in a slot of the cache
manager's state pool and starts from zero; long portions are cut into chunks that run side by side
(:func:`.gla.chunk_list`).  The reference has no recurrent mixer.
"""

from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from ..config.spec import ParamSpec, PartSpec, StateNeed
from ..errors import ConfigError
from ..kernels import ops
from .base import MIXERS, BuildEnv, Mixer, StepState
from .gla import DEFAULT_CHUNK, prepare_chunks
from .rope import shared_position


@MIXERS.register("retention")
class Retention(Mixer):
    """params: ``hidden``, ``n_heads``, ``head_dim`` (keys and queries), ``v_head_dim``, ``decay`` (a number per head),
    ``position`` (PartSpec of a rotary encoding, or none), ``eps`` (of the output norm), ``chunk`` (tokens per chunk of a long
    portion), ``init_std``."""

    graph_safe = False  # running a step twice would advance the state twice
    graph_recordable = True  # everything a step does is decided on the device

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden"])
        self.n_heads = int(spec["n_heads"])
        self.head_dim = int(spec["head_dim"])
        self.v_dim = int(spec.get("v_head_dim") or self.head_dim)
        self.decay = tuple(float(x) for x in spec["decay"])
        self.eps = float(spec.get("eps", 1e-6))
        self.chunk = int(spec.get("chunk", DEFAULT_CHUNK))
        if self.n_heads < 1 or not 1 <= self.head_dim <= 256 or self.v_dim < 1 or self.chunk < 1:
            raise ConfigError("retention: heads, head sizes (keys at most 256) and chunk must be positive")
        if len(self.decay) != self.n_heads:
            raise ConfigError(f"retention: {len(self.decay)} decays for {self.n_heads} heads")
        self.position = shared_position(spec.get("position") or PartSpec("none"), env)
        self.rotary_dim = int(getattr(self.position, "rotary_dim", 0))
        if self.rotary_dim > self.head_dim:
            raise ConfigError("retention: rotary_dim exceeds head_dim")
        H, D, Dv = self.n_heads, self.head_dim, self.v_dim
        self.k_row = H * D
        self.v_row = 2 * H * D
        self.g_row = self.v_row + H * Dv
        self.proj_rows = self.g_row + H * Dv
        self._decay: Optional[torch.Tensor] = None
        self._ones: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        std = self.spec.get("init_std")  # spread of random weights: (projections of the input, output projection)
        std_in, std_out = (float(std[0]), float(std[1])) if std else (0.02, 0.02)
        return {"in_proj.weight": ParamSpec((self.proj_rows, self.hidden), init=("normal", 0.0, std_in)),
                "o_proj.weight": ParamSpec((self.hidden, self.n_heads * self.v_dim), init=("normal", 0.0, std_out))}

    def bind(self, tensors) -> None:
        super().bind(tensors)
        self._decay = torch.tensor(self.decay, dtype=torch.float32, device=self.env.device)
        self._ones = torch.ones(self.v_dim, dtype=torch.float32, device=self.env.device)  # the output norm has no weight

    def cache_need(self):
        return StateNeed((("s", (self.n_heads, self.head_dim, self.v_dim), "float32"),))

    def max_chunks(self, n_tokens: int) -> int:
        return n_tokens // self.chunk + self.env.max_decode_rows + 1

    def workspace_bytes(self, n_tokens: int) -> int:
        item = 4 if self.env.dtype == torch.float32 else 2
        H, D, Dv = self.n_heads, self.head_dim, self.v_dim
        rows = n_tokens * ((self.proj_rows + H * Dv + self.hidden) * item + H * Dv * 4)
        return rows + self.max_chunks(n_tokens) * H * D * (Dv + 1) * 4

    def prepare(self, builder) -> None:
        self._step_lists = prepare_chunks(builder, self.chunk)

    def forward(self, h: torch.Tensor, step: StepState, cache: Any, writes_cache: bool) -> torch.Tensor:
        if not writes_cache:
            raise ConfigError("retention: a state cannot be shared between layers")
        T = h.shape[0]
        ws, dt, cap = self.env.workspace, self.env.dtype, self.env.max_step_tokens
        H, D, Dv = self.n_heads, self.head_dim, self.v_dim
        proj = ws.get("retention.proj", (T, self.proj_rows), dt, (cap, self.proj_rows))
        ops.linear(h, self.params["in_proj.weight"], proj)
        name, n_chunks, single, multi = self._step_lists
        tensors = step.extras["tensors"]
        carry = decay = None
        if multi:
            most = self.max_chunks(cap)
            carry = ws.get("gla.carry", (n_chunks, H, D, Dv), torch.float32, (most, H, D, Dv))
            decay = ws.get("gla.decay", (n_chunks, H, D), torch.float32, (most, H, D))
        o32 = ws.get("retention.o32", (T, H, Dv), torch.float32, (cap, H, Dv))
        ops.gla_scan(proj[:, : self.k_row], proj[:, self.k_row: self.v_row], proj[:, self.v_row: self.g_row], None, None,
                     1.0, D ** -0.5, cache.tensors["s"], step.state_slots, step.seg_info, len(step.segments), tensors[name],
                     n_chunks, tensors[name + ".segments"], single, multi, carry, decay, o32, a_head=self._decay,
                     rope_table=self.position.table(), neighbours=bool(getattr(self.position, "interleaved", False)))
        o = ws.get("retention.o", (T, H, Dv), dt, (cap, H, Dv))
        ops.gated_heads(o32, proj[:, self.g_row:], o, Dv, "silu", self._ones, self.eps)
        out = ws.get("retention.out", (T, self.hidden), dt, (cap, self.hidden))
        ops.linear(o.view(T, H * Dv), self.params["o_proj.weight"], out)
        return out
