"""A token embedding whose rows are layer-normed before they enter the stream."""

from __future__ import annotations

from .base import Embedding, TensorRequest, register_embedding


class NormedTokenEmbedding(Embedding):
    """``x = layer_norm(table[token]) * norm_weight (+ norm_bias)``, gather and norm in one launch.

    The same launch leaves the copy the model asks for (``keep``) and, when the block that runs
    first takes its norm from the launch before it, the rows of that norm."""

    keeps_output = True

    def __init__(self, *, vocab_size: int, width: int, table: str, eps: float, norm_weight: str,
                 norm_bias: str | None = None):
        self.vocab, self.width, self.name, self.eps = vocab_size, width, table, float(eps)
        self.wn, self.bn = norm_weight, norm_bias

    def tensor_requests(self):
        req = {self.name: TensorRequest((self.vocab, self.width), "table"),
               self.wn: TensorRequest((self.width,), "vector")}
        if self.bn:
            req[self.bn] = TensorRequest((self.width,), "vector")
        return req

    def bind(self, tensors):
        self.table, self.weight = tensors[self.name], tensors[self.wn]
        self.bias = tensors[self.bn] if self.bn else None

    def forward(self, ctx, x, position, keep=None):
        if position.embedding_table() is not None:
            raise ValueError("a normed token embedding takes no position table")
        more = {}
        nxt = getattr(ctx, "next_block", None)
        if getattr(nxt, "takes_norm_ahead", False):
            ahead = getattr(nxt.norm1, "row_norm", None)
            if ahead is not None:
                more = dict(out=ctx.buffer("normed", x.shape, ctx.dtype), norm=ahead())
        ctx.ops.embed_norm(x, ctx.tok_ids, ctx.tok_req, self.table, self.weight, self.bias, self.eps,
                           ctx.status, feedback=ctx.feedback, keep=keep, **more)
        ctx.normed_ahead = bool(more)


register_embedding("normed_token_table", NormedTokenEmbedding)
