"""Two mixers side by side on the same input, and the per-layer token input.

`ParallelMixer` hands both results on as `ops.functional.Branches`: how they are weighted and whether each is RMS-normalised first is part of
the step that adds them to the residual stream (`ops.functional.residual_join`), one kernel at inference. There, too, everything that
reads the common input is one product.
"""
from __future__ import annotations

import torch

from ..ops import functional as F
from .blocks import Builder, Norm, back_to_back


class ParallelMixer:
  """`join` = (left factor, right factor, normalise each result first)."""

  def __init__(self, b: Builder, config, name: str, build_left, build_right, join: tuple):
    c = config
    ab = b.sub(*name.split("/"))
    self.left, self.right, self.factors = build_left(ab, "left"), build_right(ab, "right"), (float(join[0]), float(join[1]))
    self.norms = tuple(Norm(ab, n, c.emb_dim, c.normalization_layer_epsilon) if join[2] else None for n in ("left_norm", "right_norm"))
    self.parts = self.left.in_parts + self.right.in_parts
    self.fused = back_to_back(ab, self.parts)

  def __call__(self, x, ctx):
    cache = ctx.cache
    caches = (cache.left, cache.right) if cache is not None else (None, None)
    ctx.cache = caches[0]
    rows = None
    if self.fused is not None and self.left.serves(x, ctx) and self.right.serves(x, ctx) and self.fused.fusable():
      rows = torch.split(F.linear(x, self.fused).view(x.shape[0] * x.shape[1], -1), self.fused.rows, dim=-1)
    n = len(self.left.in_parts)
    left = self.left(x, ctx, rows=rows[:n] if rows is not None else None, out_bias=False)
    ctx.cache = caches[1]
    right = self.right(x, ctx, rows=rows[n:] if rows is not None else None)
    ctx.cache = cache
    return F.Branches([F.Branch(left, self.left.bo, self.norms[0], self.factors[0]), F.Branch(right, None, self.norms[1], self.factors[1])])


class TokenSide:
  """A second embedding of the tokens, `dim` numbers per layer, that joins the stream after the feed-forward: tanh-GELU of a projection of
  the stream gates it, a projection brings it to the model width, an RMS norm with a weight closes it."""

  def __init__(self, b: Builder, config, dim: int):
    c = config
    sb = b.sub("token_side")
    self.embedding = sb.table("embedding", (c.vocab_size, dim), ("vocab", "embed_vocab"))
    self.gate = sb.sub("gate").linear("kernel", (c.emb_dim,), (dim,), ("embed", "mlp"))
    self.proj = sb.sub("proj").linear("kernel", (dim,), (c.emb_dim,), ("mlp", "embed"))
    self.norm = Norm(sb, "norm", c.emb_dim, c.normalization_layer_epsilon)

  def __call__(self, h, ctx):
    """h [B, S, D]: the stream in the compute type -> the branch before its norm."""
    return F.linear(F.token_gate(F.linear(h, self.gate), self.embedding, ctx.tokens), self.proj)
