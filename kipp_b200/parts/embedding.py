"""Token embedding and output head.

x_t = float(E[id_t, :]), times ``scale`` where given (src/kipp.c:2940-2942); logits = W_lm n
for the wanted rows only, W_lm being the embedding when tied
(src/kipp.c:951-956, 3013-3018).  The parts themselves: csrc/host/parts.hpp."""
from __future__ import annotations

from typing import Optional

from .base import EmbeddingStage, Part


class TokenEmbedding(EmbeddingStage):
    kind = "token_embedding"

    def __init__(self, vocab_size: int, hidden_size: int, weight_name: str = "weight", scale: float = 1.0):
        self.scale = float(scale)
        self.vocab_size = vocab_size
        self.hidden_size = hidden_size
        self.weight_name = weight_name

    def params(self, prefix, ctx) -> dict:
        return {"vocab_size": self.vocab_size, "hidden_size": self.hidden_size, "weight_name": self.weight_name,
                "scale": self.scale}


class TokenSideTable(EmbeddingStage):
    """A second table [vocab, cols] that layers read by token, each its own columns (``TokenSide``)."""
    kind = "token_side_table"

    def __init__(self, vocab_size: int, cols: int, weight_name: str = "weight"):
        self.vocab_size, self.cols, self.weight_name = vocab_size, cols, weight_name

    def params(self, prefix, ctx) -> dict:
        return {"vocab_size": self.vocab_size, "cols": self.cols, "weight_name": self.weight_name}


class TokenSide(Part):
    """What a layer's own embedding e of the token adds to the stream: x += rmsnorm(W_proj (gelu(W_gate x) * e))
    with e the columns [offset, offset + dim) of the token's row of ``table`` (a ``TokenSideTable`` of
    ``table_cols`` columns)."""
    kind = "token_side"

    def __init__(self, vocab_size: int, hidden_size: int, dim: int, table: str, table_cols: int, offset: int, eps: float,
                 names: Optional[dict] = None):
        self.vocab_size, self.hidden_size, self.dim, self.table, self.table_cols = vocab_size, hidden_size, dim, table, table_cols
        self.offset, self.eps, self.names = offset, float(eps), dict(names or {})

    def params(self, prefix, ctx) -> dict:
        return {"vocab_size": self.vocab_size, "hidden_size": self.hidden_size, "dim": self.dim, "table": self.table,
                "table_cols": self.table_cols, "offset": self.offset, "eps": self.eps, "names": self.names}


class OutputHead(Part):
    """``tied_to`` names the checkpoint tensor (an embedding matrix) that stands
    in when the checkpoint has no head of its own."""
    kind = "output_head"

    def __init__(self, vocab_size: int, hidden_size: int, tied_to: Optional[str] = None, weight_name: str = "weight",
                 logit_scale: float = 1.0, logit_softcap: float = 0.0):
        self.vocab_size = vocab_size
        self.hidden_size = hidden_size
        self.tied_to = tied_to
        self.weight_name = weight_name
        # logits * logit_scale, then (logit_softcap c > 0) c tanh(logits / c)
        self.logit_scale, self.logit_softcap = float(logit_scale), float(logit_softcap)

    def params(self, prefix, ctx) -> dict:
        return {"vocab_size": self.vocab_size, "hidden_size": self.hidden_size, "tied_to": self.tied_to,
                "weight_name": self.weight_name, "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap}
