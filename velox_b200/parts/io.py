"""The two ends of a model: token embedding and the language-model head
(src/transformer.py:27,44 and 60-68 of the reference)."""
from __future__ import annotations

import torch

from ..ops import kernels
from ..ops.linear import linear, use_tensor_core_kernel
from .base import Part, StateSpec
from .registry import register_part


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    """``resid[t] = table[ids[t]] * scale``, widened to the float32 residual stream (``scale``: 1).

    ``bigram`` ({buckets, mul_prev, mul_cur}; weight ``bigram`` [buckets + 1, width]): row ``(previous token * mul_prev +
    token * mul_cur) mod buckets`` of a second table is added, its last row for a sequence's first token.  The
    previous token of a request is a state row of the embedding (int32)."""

    def __init__(self, params, weights, dtype, device) -> None:
        super().__init__(params, weights, dtype, device)
        self.vocab_size = int(params["vocab_size"])
        self.hidden_size = int(params["hidden_size"])
        self.scale = float(params.get("scale", 1.0))
        self.table = self.expect("weight", (self.vocab_size, self.hidden_size))
        self.pairs = None
        if params.get("bigram"):
            b = params["bigram"]
            self.mul_prev, self.mul_cur = int(b["mul_prev"]), int(b["mul_cur"])
            self.pairs = self.expect("bigram", (int(b["buckets"]) + 1, self.hidden_size))
            kernels.heads()

    def state_needs(self):
        return None if self.pairs is None else StateSpec((1,), torch.int32)

    def forward(self, ids, resid, ctx) -> None:
        if self.pairs is not None:
            kernels.embed_pairs(self.table, self.pairs, self.mul_prev, self.mul_cur, self.scale, ids,
                                getattr(ctx, "fed_tokens", None), ctx.positions, ctx.embedding_state, resid, ctx.q_start,
                                ctx.q_len, ctx.seq_slots, ctx.num_seqs, ctx.num_tokens, ctx.status)
            return
        # ctx.fed_tokens: the sampler's tokens of the step before, for ids that name one of them.
        kernels.embed(self.table, ids[: ctx.num_tokens], resid, ctx.status, getattr(ctx, "fed_tokens", None),
                      self.scale)


@register_part("lm_head", "linear_head")
class LinearHead(Part):
    """``logits = x @ W.T`` without bias, returned in float32; with a ``softcap`` parameter c the
    logits become ``c * tanh(logits / c)``."""

    def __init__(self, params, weights, dtype, device) -> None:
        super().__init__(params, weights, dtype, device)
        self.vocab_size = int(params["vocab_size"])
        self.hidden_size = int(params["hidden_size"])
        self.weight = self.expect("weight", (self.vocab_size, self.hidden_size))
        cap = params.get("softcap")
        self.softcap = None if cap is None else float(cap)
        if self.softcap is not None and not self.softcap > 0.0:
            raise ValueError(f"softcap must be positive, got {self.softcap}")

    def forward(self, x, num_rows, ctx) -> torch.Tensor:
        logits = self._project(x, num_rows, ctx)
        if self.softcap is not None:
            kernels.softcap(logits, num_rows, self.softcap)
        return logits

    def _project(self, x, num_rows, ctx) -> torch.Tensor:
        ws = ctx.workspace
        logits = ws.get("lm_head.logits", (ws.max_logit_rows, self.vocab_size), torch.float32)
        if self.dtype == torch.float32:
            linear(x, self.weight, None, logits, num_rows)
        elif use_tensor_core_kernel(x, self.weight, num_rows):
            # float32 logits straight from the accumulators
            linear(x, self.weight, None, logits, num_rows, status=ctx.status)
        else:
            low = ws.get("lm_head.logits_lowp", (ws.max_logit_rows, self.vocab_size), self.dtype)
            linear(x, self.weight, None, low, num_rows)
            kernels.cast_bf16_to_f32(low, logits, num_rows * self.vocab_size)
        return logits[:num_rows]
