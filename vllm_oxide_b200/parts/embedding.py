"""Token embedding (row gather into the float32 residual, crates/engine/src/backend/cpu/mod.rs:172-180)
and the output head (logits = normed x E^T in float32; E is the embedding table when the
configuration ties them, crates/engine/src/model.rs:344)."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from .. import kernels
from ..tuning import TUNING
from .base import FoldedState, StateSpec, StepContext
from .linear import to_compute


@dataclass(frozen=True, eq=False)
class PairVectors:
    """A vector for every pair of neighbouring tokens: row (previous * mul_prev + token * mul_cur) mod (rows - 1) of `table`, the
    last row for a sequence's first token."""
    table: torch.Tensor
    mul_prev: int
    mul_cur: int


class Embedding:
    def __init__(self, table: torch.Tensor, dtype=torch.bfloat16, device="cuda", scale: float = 1.0,
                 positions: torch.Tensor = None, pairs: Optional[PairVectors] = None, keep: Optional[str] = None):
        """`scale`: every row is multiplied by it on its way into the float32 residual. `positions` [max positions,
        hidden]: a learned vector per position, added (not scaled) to the token's row. `pairs`: a vector per pair of neighbouring
        tokens, added likewise; the last token of a request's step is then part of the request's state (`state_spec`). `keep`: the
        float32 step buffer in which a copy of the result is left for later layers."""
        self.table = to_compute(table, dtype, device)
        if positions is not None and (positions.dim() != 2 or positions.shape[1] != table.shape[1]):
            raise ValueError(f"position table {list(positions.shape)} does not fit a width of {table.shape[1]}")
        self.pos_table = to_compute(positions, dtype, device) if positions is not None else None
        if pairs is not None and (pairs.table.dim() != 2 or pairs.table.shape[1] != table.shape[1] or pairs.table.shape[0] < 2):
            raise ValueError(f"a table of {list(pairs.table.shape)} vectors of pairs does not fit a width of {table.shape[1]}")
        self.pairs = (to_compute(pairs.table, dtype, device), int(pairs.mul_prev), int(pairs.mul_cur)) if pairs is not None else None
        self.keep = keep
        self.scale = float(scale)
        self.vocab, self.hidden = self.table.shape
        self.err_flag = torch.zeros(1, dtype=torch.int32, device=device)

    def kernel_modules(self, dtype, max_rows):
        return ("elementwise",)

    def state_spec(self) -> Optional[StateSpec]:
        """The last token of each request's previous step, where the embedding of a token needs the one before it."""
        return StateSpec((1,), torch.int32) if self.pairs is not None else None

    def can_fold(self) -> bool:
        return self.pairs is None and self.keep is None and self.pos_table is None and self.scale == 1.0

    def forward(self, ctx: StepContext, state: Optional[torch.Tensor] = None) -> torch.Tensor:
        resid = ctx.alloc((ctx.rows, self.hidden), torch.float32)
        if self.pairs is not None or self.keep is not None:
            pairs = None
            if self.pairs is not None:
                pairs = self.pairs + (ctx.row_seq, ctx.seq_starts, ctx.state_slots, state)
            kernels.embed_pairs(self.table, ctx.tokens, resid, ctx.positions, self.err_flag, self.scale, self.pos_table, pairs,
                                ctx.shared[self.keep] if self.keep is not None else None)
            return resid
        kernels.embed(self.table, ctx.tokens, resid, self.err_flag, self.scale, self.pos_table,
                      ctx.positions if self.pos_table is not None else None)
        return resid

    def forward_folded(self, ctx: StepContext, next_norm) -> FoldedState:
        """The embedding with the first norm's input prepared (see FoldedState)."""
        h = self.hidden
        st = FoldedState(resid=ctx.alloc((ctx.rows, h), torch.float32), xn=ctx.alloc((ctx.rows, h), torch.bfloat16),
                         ssq=ctx.alloc((-(-h // 128), TUNING.few_rows), torch.float32))
        kernels.embed_fold(self.table, ctx.tokens, st.resid, next_norm.weight, st.xn, st.ssq, self.err_flag)
        return st


class LMHead:
    """`weight` may be the Embedding's own table (tied): no copy is made then."""

    def __init__(self, weight: torch.Tensor):
        self.weight = weight
        self.vocab, self.hidden = weight.shape

    def weight_bytes(self) -> int:
        return self.weight.numel() * self.weight.element_size()

    def kernel_modules(self, dtype, max_rows):
        return ("gemm_f32",) if dtype == torch.float32 else ("gemm_sm100",)

    def forward(self, normed: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
        kernels.linear(normed, self.weight, out)
        return out

    def can_fold(self) -> bool:
        return self.weight.dtype == torch.bfloat16 and self.hidden % 8 == 0

    def forward_folded(self, st: FoldedState, eps: float, rows: int, out: torch.Tensor) -> torch.Tensor:
        """Logits of the first `rows` rows straight from the folded residual: the final norm is the
        per-token scale of the product."""
        kernels.gemm_fused(st.xn[:rows], self.weight, out, kernels.EPI_STORE, self.vocab, ssq_in=st.ssq, eps=eps)
        return out

    def pick_folded(self, st: FoldedState, eps: float, rows: int, temperature, seeds, steps, part_val: torch.Tensor,
                    part_idx: torch.Tensor, nan_flags: torch.Tensor, out: torch.Tensor, also=()) -> None:
        """Tokens of the first `rows` rows straight from the folded residual, without the logits ever
        going to memory: the head product's epilogue leaves the best (value, index) pair of every
        128 logits, a second small kernel reduces a row's pairs. Same picks as `forward_folded`
        followed by `kernels.pick_tokens` (the same values, compared by the same rule). `also`: further
        places the tokens are written to (see `kernels.pick_final`)."""
        kernels.gemm_fused(st.xn[:rows], self.weight, None, kernels.EPI_PICK, self.vocab, ssq_in=st.ssq, eps=eps,
                           pick=(temperature, seeds, steps, part_val, part_idx, nan_flags))
        kernels.pick_final(part_val, part_idx, rows, self.vocab, nan_flags, out, also)
