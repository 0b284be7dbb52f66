"""
Embeddings beside the token embedding.

`PairEmbedding`: a row by the pair (previous token, token), added to the scaled token embedding as it starts
the residual stream.  The row is (previous * mul_prev + token * mul_cur) mod buckets, the table's last row for
a request's first token.  The kernel that gathers the token embedding gathers this row too; inside a step the
previous token is the one before in the batch, ahead of a step's first token it is the last one the cache
manager has on record for the request (`StepContext.prev_tokens`).
"""

from __future__ import annotations

import torch

from tinyserve_llm_b200.config.spec import PairEmbeddingSpec
from tinyserve_llm_b200.parts.base import Part, Runtime, TensorDecl, register_part


@register_part("embedding", "pair_embedding")
class PairEmbedding(Part):
    role = "embedding"
    graph_safe = True

    @classmethod
    def declare(cls, spec: PairEmbeddingSpec) -> dict[str, TensorDecl]:
        if spec.buckets <= 0 or spec.size <= 0 or spec.mul_prev < 0 or spec.mul_cur < 0:
            raise ValueError(f"a pair embedding of {spec.buckets} rows of {spec.size} with multipliers {spec.mul_prev} and {spec.mul_cur}")
        return {spec.name: TensorDecl((spec.buckets + 1, spec.size))}

    def __init__(self, spec: PairEmbeddingSpec, tensors: dict[str, torch.Tensor], rt: Runtime) -> None:
        super().__init__(spec, tensors, rt)
        self.table = tensors[spec.name].to(device=rt.device, dtype=rt.dtype).contiguous()
