"""Token embedding (a row copy, src/qwen.ts:162-163; ``scale`` multiplies the rows when a model asks for it) and the output head
(logits = W h, no bias; W is the embedding matrix itself when tied: src/qwen.ts:152,203).
With ``scale`` the head's logits are multiplied by it, with ``softcap`` they then become softcap * tanh(logits / softcap)."""
from __future__ import annotations

import torch

from .. import kernels
from .base import Part, StateSpec, TensorDecl, WeightSource, register_part
from .linear import Linear


@register_part("embedding", "token_embedding")
class TokenEmbedding(Part):
    def __init__(self, prefix: str, vocab_size: int, hidden_size: int, name: str = "embed_tokens", suffix: str = ".weight",
                 scale: float = 1.0):
        self.vocab_size, self.hidden_size, self.scale = vocab_size, hidden_size, float(scale)
        self.tensor_name = f"{prefix}{name}{suffix}"
        self.table = None
        self.runtime = None

    def tensor_decls(self):
        return [TensorDecl(self.tensor_name, (self.vocab_size, self.hidden_size))]

    def load(self, source: WeightSource):
        self.table = source.matrix(self.tensor_name)
        self.runtime = source.runtime

    def state_spec(self):
        return None

    def forward(self, token_ids: torch.Tensor, ctx=None, state=None) -> torch.Tensor:
        x = torch.empty((token_ids.numel(), self.hidden_size), dtype=torch.float32, device=token_ids.device)
        kernels.embed(self.table, token_ids, x, self.runtime.status, scale=self.scale)
        return x


@register_part("embedding", "token_pair_embedding")
class TokenPairEmbedding(TokenEmbedding):
    """The token's row times ``scale`` plus a row of a second table that the last two tokens choose:
    (previous * mul_prev + token * mul_cur) mod ``buckets``; a sequence's first token takes the table's last row (number
    ``buckets``).  A request's last token is its state: int32 [1] in its slot."""

    def __init__(self, prefix: str, vocab_size: int, hidden_size: int, buckets: int, mul_prev: int, mul_cur: int,
                 pair_name: str = "bigram", **base):
        super().__init__(prefix, vocab_size, hidden_size, **base)
        if buckets <= 0:
            raise ValueError("token_pair_embedding: the table of pairs needs at least one row beside the first token's")
        self.buckets, self.mul_prev, self.mul_cur = int(buckets), int(mul_prev), int(mul_cur)
        self.pair_name = prefix + pair_name
        self.pairs = None

    def tensor_decls(self):
        return super().tensor_decls() + [TensorDecl(self.pair_name, (self.buckets + 1, self.hidden_size))]

    def load(self, source: WeightSource):
        super().load(source)
        self.pairs = source.matrix(self.pair_name)

    def state_spec(self):
        return StateSpec(shape=(1,), dtype=torch.int32)

    def forward(self, token_ids: torch.Tensor, ctx=None, state=None) -> torch.Tensor:
        if ctx is None or state is None:
            raise RuntimeError("token_pair_embedding: the previous tokens live in the requests' state slots")
        x = torch.empty((token_ids.numel(), self.hidden_size), dtype=torch.float32, device=token_ids.device)
        kernels.embed_pairs(self.table, self.pairs, ctx, state, x, self.scale, self.mul_prev, self.mul_cur, self.runtime.status)
        return x


@register_part("head", "lm_head")
class LMHead(Part):
    def __init__(self, prefix: str, vocab_size: int, hidden_size: int, tied_to: str | None = None,
                 name: str = "lm_head", suffix: str = ".weight", softcap: float | None = None,
                 any_inner_size: bool = False, scale: float = 1.0):
        if softcap is not None and not softcap > 0:
            raise ValueError("lm_head: softcap must be positive")
        self.vocab_size, self.hidden_size = vocab_size, hidden_size
        self.softcap = None if softcap is None else float(softcap)
        self.any_inner_size, self.scale = any_inner_size, float(scale)
        self.tensor_name = f"{prefix}{tied_to or name}{suffix}"
        self.tied = tied_to is not None
        self.linear = None

    def tensor_decls(self):
        return [] if self.tied else [TensorDecl(self.tensor_name, (self.vocab_size, self.hidden_size))]

    def load(self, source: WeightSource):
        self.linear = Linear(source.matrix(self.tensor_name), None, source.runtime.status, any_inner_size=self.any_inner_size)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        logits = self.linear.forward(h, out_dtype=torch.float32)
        if self.softcap is not None or self.scale != 1.0:
            kernels.softcap(logits, self.softcap or 0.0, factor=self.scale)
        return logits
