"""Token embedding and output head."""
from __future__ import annotations

from ..kernels import ops
from .base import Part, StateRequirement, TensorSpec
from .linear import Linear
from .spec import register_part


class TokenEmbedding(Part):
    """x[t,:] = E[token[t],:] * scale in float32; scale 1 in the plain case
    (crates/forward/src/core/composites/embed.rs:26-62).  The tensor is `<prefix><weight_name>`.

    `pairs` (optional: buckets, mul_prev, mul_cur, weight_name): a second table of buckets + 1 rows of which every
    token takes the row (mul_prev * token before + mul_cur * token) mod buckets, and a request's first token the last
    one; it is added as it is.  The token before is kept in the request's state slot from step to step (one int32, the
    id + 1)."""
    graph_safe = True
    category = "embedding"

    def __init__(self, runtime=None, prefix="", *, vocab: int, width: int, init_std: float = 0.02,
                 scale: float = 1.0, weight_name: str = "weight", pairs: dict | None = None):
        super().__init__(runtime, prefix)
        self.vocab, self.width, self.init_std = int(vocab), int(width), init_std
        self.scale, self.weight_name = float(scale), weight_name
        self.pairs = dict(pairs) if pairs else None
        if self.pairs and int(self.pairs["buckets"]) < 1:
            raise ValueError("embedding of pairs: at least one bucket wanted")
        self.table = self.pair_table = None

    def state_requirement(self):
        return StateRequirement((1,), "int32") if self.pairs else None

    def own_tensor_specs(self):
        specs = {self.prefix + self.weight_name: TensorSpec((self.vocab, self.width), init=("normal", self.init_std))}
        if self.pairs:
            specs[self.prefix + self.pairs["weight_name"]] = TensorSpec(
                (int(self.pairs["buckets"]) + 1, self.width), init=("normal", self.init_std))
        return specs

    def own_bind(self, tensors):
        self.table = tensors[self.prefix + self.weight_name]
        if self.pairs:
            self.pair_table = tensors[self.prefix + self.pairs["weight_name"]].to(self.table.dtype).contiguous()

    def own_weights(self):
        return []          # a step reads n rows of the table, not the table

    def forward(self, ctx, token_ids, x, state=None):
        """state: what the cache manager keeps for this part (only where state_requirement asks for it)."""
        if self.pairs:
            ops.embedding_pairs(self.table, self.pair_table, self.pairs["mul_prev"], self.pairs["mul_cur"], token_ids,
                                ctx.batch, state, x, self.runtime.status, self.scale)
            return
        ops.embedding(self.table, token_ids, x, self.runtime.status, self.scale)


class LMHead(Part):
    """logits = h W^T (times `scale`) in float32, for the wanted rows only; a tied head reuses
    the embedding table (crates/forward/src/core/composites/output_head.rs:90-132;
    crates/models/qwen35-v2/src/loader.rs:219-223).  `softcap` (> 0): every logit passes cap * tanh(logit / cap)."""
    graph_safe = True
    category = "head"

    def __init__(self, runtime=None, prefix="", *, vocab: int, width: int, tied_to: str | None = None,
                 init_std: float = 0.02, weight_name: str = "weight", scale: float = 1.0, softcap: float = 0.0):
        super().__init__(runtime, prefix)
        self.softcap = float(softcap or 0.0)
        if self.softcap < 0.0:
            raise ValueError(f"output head: softcap = {softcap} must be positive (0 or None: none)")
        self.vocab, self.width, self.tied_to, self.init_std = int(vocab), int(width), tied_to, init_std
        self.weight_name, self.scale = weight_name, float(scale)
        self.proj = None

    def own_tensor_specs(self):
        return {self.prefix + self.weight_name: TensorSpec((self.vocab, self.width), init=("normal", self.init_std),
                                                           alias_of=self.tied_to)}

    def own_bind(self, tensors):
        self.proj = Linear(tensors[self.prefix + self.weight_name])

    def own_weights(self):
        return [self.proj.weight]

    def forward(self, ctx, h_rows, logits):
        self.proj(ctx, h_rows, logits)
        if self.scale != 1.0:
            logits.mul_(self.scale)          # float32, the wanted rows only
        if self.softcap:
            ops.softcap_rows(logits, self.softcap)


register_part("embedding", "token_embedding", TokenEmbedding)
register_part("head", "lm_head", LMHead)
