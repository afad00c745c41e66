"""The two ends of a model: token embedding and output head.

``token_embedding`` (python/freetoken/layers/embedding.py:40-57, ``embed_scale=None`` in
python/freetoken/models/minimax_m3/model.py:67-70,76): a pure row gather of ``[vocab, hidden]``
into the 32-bit residual stream, without scaling.

``linear_head`` (python/freetoken/layers/embedding.py:103-113): ``logits = y W^T`` without a bias,
kept as the float32 accumulator of the library product (the reference rounds the logits to
bfloat16 and widens them again for sampling, python/freetoken/engine/sample.py:80).  A tied head
multiplies by the embedding table and owns no tensor; a stray ``lm_head.weight`` in the file is
then ignored (embedding.py:81-90).

Other embeddings (scaled, with added position rows) and heads (bias, soft-cap, several outputs)
are other kinds in the same registries; the model asks for them by ``spec.embedding.kind`` and
``spec.head.kind``.
"""

from __future__ import annotations

from typing import Any, Dict, Optional

import torch

from ..config.spec import ParamSpec, PartSpec
from ..errors import ConfigError
from ..kernels import ops
from .base import EMBEDDINGS, HEADS, NORMS, BuildEnv, Embedding, GatedSum, Head, Part, as_rows


@EMBEDDINGS.register("token_embedding")
class TokenEmbedding(Embedding):
    """params: ``vocab``, ``hidden``, ``init_std`` (spread of random weights, 0.02), ``scale`` (1.0: the rows
    are multiplied by it in 32 bits as they enter the stream), ``norm`` (None, or the PartSpec of an RMS norm that the
    rows pass in 32 bits, with a weight under ``norm``)."""

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.vocab = int(spec["vocab"])
        self.hidden = int(spec["hidden"])
        self.init_std = float(spec.get("init_std", 0.02))
        self.scale = float(spec.get("scale", 1.0))
        self.norm = NORMS.build(spec["norm"], env) if spec.get("norm") is not None else None

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {"weight": ParamSpec((self.vocab, self.hidden), init=("normal", 0.0, self.init_std))}

    def children(self) -> Dict[str, Part]:
        return {"norm": self.norm} if self.norm is not None else {}

    def forward(self, token_ids: torch.Tensor, residual: torch.Tensor) -> None:
        ops.embedding_gather(self.params["weight"], token_ids, residual)
        if self.scale != 1.0:
            ops.scale_(residual, self.scale)
        if self.norm is not None:
            self.norm.norm_stream(residual)

    def table(self) -> torch.Tensor:
        return self.params["weight"]


@HEADS.register("linear_head")
class LinearHead(Head):
    """params: ``vocab``, ``hidden``, ``tied`` (bool: multiply by the embedding's table), ``scale`` (1.0),
    ``softcap`` (None or c: the logits become ``c tanh(logits / c)``, after the scale)."""

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.vocab = int(spec["vocab"])
        self.hidden = int(spec["hidden"])
        self.tied = bool(spec.get("tied", False))
        self.scale = float(spec.get("scale", 1.0))  # logits are multiplied by it
        self.softcap = None if spec.get("softcap") is None else float(spec["softcap"])
        if self.softcap is not None and not self.softcap > 0:
            raise ConfigError("linear_head: a soft cap must be positive")
        self._tied_weight: Optional[torch.Tensor] = None

    def param_specs(self) -> Dict[str, ParamSpec]:
        init = ("normal", 0.0, float(self.spec.get("init_std", 0.02)))
        return {} if self.tied else {"weight": ParamSpec((self.vocab, self.hidden), init=init)}

    def tie(self, embedding: Embedding) -> None:
        w = embedding.table()
        if tuple(w.shape) != (self.vocab, self.hidden):
            raise ConfigError(f"linear_head: cannot tie to an embedding table of shape {tuple(w.shape)}")
        self._tied_weight = w

    def weight(self) -> torch.Tensor:
        return self._tied_weight if self.tied else self.params["weight"]

    def forward(self, y: torch.Tensor, logits: torch.Tensor) -> None:
        w = self.weight()
        if y.dtype == torch.float32:
            torch.matmul(y, w.t(), out=logits)
        else:
            torch.mm(y, w.t(), out=logits, out_dtype=torch.float32)
        if self.scale != 1.0:
            ops.scale_(logits, self.scale)
        if self.softcap is not None:
            ops.softcap_(logits, self.softcap)


@EMBEDDINGS.register("pass_vectors")
class PassVectors(Embedding):
    """One ``[hidden]`` vector per pass of a repeated range of layers, added to every token of the
    stream before the pass (``table [passes, hidden]``, kept in 32-bit).  It is an embedding of the pass
    number rather than of a token; :meth:`vector` gives the row."""

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.passes = int(spec["passes"])
        self.hidden = int(spec["hidden"])
        self.local_name = spec.get("name", "weight")

    def param_specs(self) -> Dict[str, ParamSpec]:
        return {self.local_name: ParamSpec((self.passes, self.hidden), "float32", ("normal", 0.0, 0.3), store="bfloat16")}

    def vector(self, i: int) -> torch.Tensor:
        return self.params[self.local_name][i]

    def table(self) -> torch.Tensor:
        return self.params[self.local_name]


@EMBEDDINGS.register("stream_mix")
class StreamMix(Embedding):
    """What a repeated range of layers reads at the start of a pass: ``r <- W [r ; x0]`` with the stream ``r`` and the
    embedding output ``x0`` (``weight [hidden, 2 hidden]``, the stream's columns first).  The product's operands are of the
    engine's type, its 32-bit sums are the new stream."""

    def __init__(self, spec: PartSpec, env: BuildEnv):
        super().__init__(spec, env)
        self.hidden = int(spec["hidden"])

    def param_specs(self) -> Dict[str, ParamSpec]:
        std = self.spec.get("init_std")
        return {"weight": ParamSpec((self.hidden, 2 * self.hidden),
                                    init=("normal", 0.0, float(std) if std else 0.02))}

    def workspace_bytes(self, n_tokens: int) -> int:
        return n_tokens * 2 * self.hidden * (4 if self.env.dtype == torch.float32 else 2)

    def _pair(self, n_tokens: int) -> torch.Tensor:
        cap = self.env.max_step_tokens
        return self.env.workspace.get("stream_mix.pair", (n_tokens, 2 * self.hidden), self.env.dtype, (cap, 2 * self.hidden))

    def keep(self, residual: torch.Tensor) -> None:
        """The stream as the embedding leaves it, for the passes of this step."""
        ops.stream_step(residual, raw_out=self._pair(residual.shape[0])[:, self.hidden:])

    def mix(self, x: Any, residual: torch.Tensor) -> None:
        """Add what the layer before left (``x``) to the stream and replace the stream by the mix."""
        pair = self._pair(residual.shape[0])
        if isinstance(x, GatedSum):
            x.fold(residual, raw_out=pair[:, : self.hidden])
        else:
            x = as_rows(x, None, residual)
            if x is not None:
                ops.stream_add_norm(residual, None, x1=x)
            ops.stream_step(residual, raw_out=pair[:, : self.hidden])
        ops.linear_f32(pair, self.params["weight"], residual)
