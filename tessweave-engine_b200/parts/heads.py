"""Output heads: normalised rows in, fp32 logits out."""
from __future__ import annotations

import torch

from ..csrc import ops
from .base import Head, Runtime, StepContext, WeightDecl, register_part
from .linear import matmul_nt


@register_part("head", "linear_head")
class LinearHead(Head):
    """logits = y @ weight.T, accumulated and stored in fp32, no bias (reference: flow_engine/model.py:204).

    With ``tied`` the matrix is the embedding's: one buffer, two users, and the checkpoint brings no
    tensor for the head (flow_engine/model.py:110-112).  Steps with few rows stream the matrix once
    through the hand-written kernels; the rest is a library product.  ``scale``: the logits are then multiplied by it;
    ``softcap`` c: and then bent into (-c, c), logits <- c tanh(logits / c); both in fp32, in one pass.
    """

    def __init__(self, runtime: Runtime, vocab: int, hidden: int, tied: torch.Tensor | None = None, weight_name: str = "weight",
                 softcap: float | None = None, scale: float = 1.0):
        super().__init__(runtime)
        if softcap is not None and not softcap > 0:
            raise ValueError("head: the cap of the logits must be positive")
        self.softcap = float(softcap) if softcap is not None else None
        self.scale = float(scale)
        if min(vocab, hidden) <= 0:
            raise ValueError("head needs a positive vocabulary and width")
        self.vocab, self.hidden = int(vocab), int(hidden)
        if tied is not None and tuple(tied.shape) != (self.vocab, self.hidden):
            raise ValueError(f"a tied head needs a [{vocab}, {hidden}] matrix, got {tuple(tied.shape)}")
        self.tied = tied is not None
        self.weight_name = weight_name        # may be empty: the tensor then carries the part's own name
        self.weight = tied if tied is not None else runtime.empty(self.vocab, self.hidden)

    def weights(self) -> list[WeightDecl]:
        return [] if self.tied else [WeightDecl(self.weight_name, (self.vocab, self.hidden), dest=self.weight)]

    def redundant_names(self) -> list[str]:
        return [self.weight_name] if self.tied else []

    def forward(self, ctx: StepContext, logits: torch.Tensor, y: torch.Tensor, n_rows: int) -> None:
        out = logits[:n_rows]
        if ops.stream_product_preferred(y, self.weight, n_rows):
            ops.gemm_tcgen05_stream(out, y, self.weight, n_rows, ctx.status)
        elif ops.small_m_supported(y, self.weight, n_rows):
            ops.gemm_small_m(out, y, self.weight, n_rows)
        else:
            matmul_nt(out, y[:n_rows], self.weight)
        if self.softcap is not None or self.scale != 1.0:
            ops.softcap(out, self.softcap, self.scale)
