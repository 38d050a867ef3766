"""Embedding tables (``/root/reference/src/tiny_llm_ref/embedding.py``)."""

from __future__ import annotations

import torch

from extensions_b200 import tiny_llm_ext_b200

from .basics import linear
from .quantize import QuantizedWeights, as_packed_i32, dequantize_weights, quantized_linear


class Embedding:
    """Dense table (embedding.py:7-23)."""

    def __init__(self, vocab_size: int, embedding_dim: int, weight: torch.Tensor):
        self.vocab_size = vocab_size
        self.embedding_dim = embedding_dim
        self.weight = weight

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        return self.weight[as_packed_i32(x).long()]

    def as_linear(self, x: torch.Tensor) -> torch.Tensor:
        return linear(x, self.weight)


class PairEmbedding:
    """The start of an fp32 residual stream over a ragged batch: ``table[token] * scale``, plus, with ``pairs [buckets + 1, D]``, a
    row for the token and the one before it, ``(previous * mul_prev + token * mul_cur) mod buckets``, the last row for a
    sequence's first token.  The token before comes from the batch or, at the start of a portion, from the request's cache
    (``RaggedPlan.seq_prev``).  The norms that read the stream first are made in the same launch."""

    def __init__(self, weight: torch.Tensor, scale: float = 1.0, pairs: torch.Tensor | None = None, buckets: int = 0, mul_prev: int = 0, mul_cur: int = 0):
        self.weight, self.scale = weight.contiguous(), float(scale)
        self.pairs = None if pairs is None else pairs.contiguous()
        self.mul_prev, self.mul_cur = int(mul_prev), int(mul_cur)
        if self.pairs is not None and tuple(self.pairs.shape) != (int(buckets) + 1, self.weight.shape[1]):
            raise ValueError("pair embedding: the table must be [buckets + 1, width]")

    def __call__(self, plan, eps: float, norm: torch.Tensor, norm2: torch.Tensor | None = None):
        """-> (x32 [T, D] fp32, the norm times ``norm``, the norm times ``norm2`` or None)."""
        from extensions_b200.tiny_llm_ext_b200 import blocks

        return blocks.embed_pairs(plan.ids, self.weight, self.scale, pairs=self.pairs, mul_prev=self.mul_prev, mul_cur=self.mul_cur, tok_pos=plan.tok_pos,
                                  tok_seq=plan.tok_seq, seq_prev=plan.seq_prev, weight=norm, weight2=norm2, eps=eps)


class QuantizedEmbedding:
    """Packed table (embedding.py:25-57): readable gather+dequantise, or the
    fused gather kernel when ``use_custom_kernel`` and biases are present."""

    def __init__(self, vocab_size: int, embedding_dim: int, weight: QuantizedWeights, use_custom_kernel: bool = False):
        self.vocab_size = vocab_size
        self.embedding_dim = embedding_dim
        self.weight = weight
        self.use_custom_kernel = use_custom_kernel

    def __call__(self, x: torch.Tensor) -> torch.Tensor:
        w = self.weight
        if not self.use_custom_kernel or w.biases is None:
            rows = as_packed_i32(x).long()
            return dequantize_weights(
                as_packed_i32(w.weight)[rows],
                w.scales[rows],
                None if w.biases is None else w.biases[rows],
                w.group_size,
                w.bits,
            )
        ids = x if x.dtype in (torch.int32, torch.uint32) else x.to(torch.int32)
        return tiny_llm_ext_b200.quantized_embedding(ids.contiguous(), w.scales, w.biases, w.weight, w.group_size, w.bits)

    def as_linear(self, x: torch.Tensor) -> torch.Tensor:
        return quantized_linear(x, self.weight)
