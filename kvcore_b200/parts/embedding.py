"""Token embedding and output head.

Embedding is a row gather (kvcore/model/models/llama3.py:161-165, 178-180).  The head
multiplies the selected hidden rows with the ``[V, E]`` matrix, shares the embedding matrix
when tied, and applies ``logit_scale`` when it is not 1 (llama3.py:219-225, 245-247;
kvcore/sample/logits_processor.py:46-54).  Logits leave the head in 32-bit; ``softcap`` bounds them smoothly,
``cap * tanh(logits * logit_scale / cap)``.
"""
from __future__ import annotations

import torch

from .. import kernels as K
from .base import EMBEDDINGS, LM_HEADS, Part, StateSpec, WeightSlot


class TokenEmbedding(Part):
    graph_safe = True

    def __init__(self, *, vocab_size: int, hidden_size: int, name: str, tensor: str | None = None,
                 scale: float | None = None, side_tensor: str | None = None, side_width: int = 0,
                 pairs: dict | None = None, norm: dict | None = None, dtype, device) -> None:
        self.vocab_size = int(vocab_size)
        self.hidden_size = int(hidden_size)
        self.name = name
        # ``scale``: the embedded tokens are ``table[id] * scale``, formed in 32-bit; the result is then the
        # first value of a 32-bit residual stream rather than rows of the activation type
        self.scale = None if scale is None else float(scale)
        self.tensor = tensor or f"{name}.weight"     # the table's full checkpoint name
        self.weight = torch.empty(self.vocab_size, self.hidden_size, dtype=dtype, device=device)
        # ``side_tensor``: a second table ``[vocab, side_width]`` whose row of a token is an input of the
        # layers themselves (each block reads its own columns); gathered once a step by ``side_rows``
        self.side_tensor, self.side_width = side_tensor, int(side_width)
        if (side_tensor is None) != (self.side_width == 0):
            raise ValueError("a side table needs both its tensor's name and its width")
        self.side_weight = (torch.empty(self.vocab_size, self.side_width, dtype=dtype, device=device)
                            if side_tensor is not None else None)

        # ``pairs`` (``dict(tensor, buckets, mul_prev, mul_cur)``): a table ``[buckets + 1, width]`` whose row
        # ``(id in front * mul_prev + id * mul_cur) mod buckets`` (the last row for a request's first token) is
        # added; the id in front of a portion is per-request state.  ``norm`` (``dict(tensor, eps, offset)``): an
        # RMS norm of the sum with the factor ``stored + offset``.  With either the result is the first value of
        # a 32-bit residual stream.
        self.pairs, self.norm = None if pairs is None else dict(pairs), None if norm is None else dict(norm)
        if (self.pairs is not None or self.norm is not None) and self.scale is not None:
            raise ValueError("a scaled embedding takes no pair table and no norm")
        self.pair_weight = self.norm_stored = self.norm_weight = None
        if self.pairs is not None:
            self.pair_weight = torch.empty(int(self.pairs["buckets"]) + 1, self.hidden_size, dtype=dtype, device=device)
        if self.norm is not None:
            self.norm_stored = torch.empty(self.hidden_size, dtype=dtype, device=device)
            self.norm_weight = torch.empty(self.hidden_size, dtype=torch.float32, device=device)

    def weight_slots(self) -> list[WeightSlot]:
        slots = [WeightSlot(self.tensor, self.weight)]
        if self.side_weight is not None:
            slots.append(WeightSlot(self.side_tensor, self.side_weight))
        if self.pairs is not None:
            slots.append(WeightSlot(self.pairs["tensor"], self.pair_weight))
        if self.norm is not None:
            slots.append(WeightSlot(self.norm["tensor"], self.norm_stored,
                                    init="zeros" if float(self.norm.get("offset", 0.0)) == 1.0 else "ones"))
        return slots

    def finalize_weights(self) -> None:
        if self.norm is not None:
            self.norm_weight.copy_(self.norm_stored.to(torch.float32) + float(self.norm.get("offset", 0.0)))

    def state_spec(self) -> StateSpec | None:
        """The request's last token id, where the embedding of the next one reads it."""
        return StateSpec((1,), torch.int32) if self.pairs is not None else None

    def forward_step(self, ctx) -> torch.Tensor:
        """The step's embedded tokens; an embedding with per-request state finds it in ``ctx.embedding_state``."""
        if self.pairs is None and self.norm is None:
            return self.forward(ctx.token_ids)
        pairs = self.pairs or {}
        return K.embed_pairs(self.weight, ctx.token_ids, pairs=self.pair_weight, mul_prev=pairs.get("mul_prev", 0),
                             mul_cur=pairs.get("mul_cur", 0), weight=self.norm_weight,
                             eps=float(self.norm["eps"]) if self.norm else 0.0,
                             state=ctx.embedding_state if self.pairs else None, ctx=ctx)

    def forward(self, token_ids: torch.Tensor) -> torch.Tensor:
        if self.scale is not None:
            return K.embed_scaled(self.weight, token_ids, self.scale)
        return K.gather_rows(self.weight, token_ids)

    def side_rows(self, token_ids: torch.Tensor) -> torch.Tensor | None:
        """The step's rows ``[T, side_width]`` of the side table (None without one)."""
        return None if self.side_weight is None else K.gather_rows(self.side_weight, token_ids)


class LMHead(Part):
    graph_safe = True

    def __init__(
        self,
        *,
        vocab_size: int,
        hidden_size: int,
        name: str,
        tied_to: str | None = None,
        logit_scale: float = 1.0,
        softcap: float | None = None,
        tied_weight: torch.Tensor | None = None,
        tensor: str | None = None,
        dtype,
        device,
    ) -> None:
        self.vocab_size = int(vocab_size)
        self.hidden_size = int(hidden_size)
        self.name = name
        self.tied_to = tied_to
        self.logit_scale = float(logit_scale)
        self.softcap = None if softcap is None else float(softcap)
        if self.softcap is not None and not self.softcap > 0:
            raise ValueError(f"the logits' cap must be positive, got {softcap}")
        self.tensor = tensor or f"{name}.weight"     # the matrix's full checkpoint name
        if tied_to is not None:
            if tied_weight is None:
                raise ValueError(f"lm head is tied to {tied_to!r} but no such matrix was given")
            self.weight = tied_weight
        else:
            self.weight = torch.empty(self.vocab_size, self.hidden_size, dtype=dtype, device=device)

    def weight_slots(self) -> list[WeightSlot]:
        if self.tied_to is not None:
            return []
        return [WeightSlot(self.tensor, self.weight)]

    def ignorable_tensor_names(self) -> list[str]:
        # a checkpoint may still carry the tied matrix under the head's own name
        return [self.tensor] if self.tied_to is not None else []

    def forward(self, hidden: torch.Tensor) -> torch.Tensor:
        logits = K.linear(hidden, self.weight, None, out_dtype=torch.float32)
        if self.softcap is not None:
            return K.softcap(logits, self.logit_scale, self.softcap)
        if self.logit_scale != 1.0:
            logits = logits * self.logit_scale
        return logits


EMBEDDINGS.register("token_embedding", TokenEmbedding)
LM_HEADS.register("lm_head", LMHead)

__all__ = ["LMHead", "TokenEmbedding"]
