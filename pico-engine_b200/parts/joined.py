"""Sublayers that read the same normed rows, run on one first and one last product."""
from __future__ import annotations

import torch

from ..ops import linear
from .base import JoinedProducts, Part


class JoinedSublayers(Part):
    """sum_i sublayer_i(h) for sublayers that can lend their first and last products (``JoinedProducts``): the first weights stacked are
    one product for all of them, each sublayer works from its columns of that product's rows into its columns of the rows of the last
    product, and that product's sum over columns adds the sublayers up in its float32 accumulator.

    Takes the weights from its members after they have taken theirs.  ``active`` says whether it did: members that cannot join, or
    weights of different dtypes, stay as they are."""

    def __init__(self, members, dtype, device):
        super().__init__(None, dtype, device)
        self.members, self.active = tuple(members), False
        self.w_in = self.w_out = None
        self.cols, self.side_cols, self.padded = [], [], False

    def take_tensors(self, get):
        if not all(isinstance(m, JoinedProducts) and m.can_join() for m in self.members):
            return
        if len({t.dtype for m in self.members for t in m.weights() if t.dim() == 2}) != 1:
            return
        firsts, lasts = [], []
        for m in self.members:
            first, last = m.lend_products()
            self.cols.append(sum(t.shape[0] for t in firsts))
            self.side_cols.append(sum(t.shape[1] for t in lasts))
            pad, side_pad = -first.shape[0] % 8, -last.shape[1] % 8          # every sublayer's columns start at a multiple of 8
            firsts += [first] + ([first.new_zeros(pad, first.shape[1])] if pad else [])
            lasts += [last] + ([last.new_zeros(last.shape[0], side_pad)] if side_pad else [])
            self.padded |= side_pad > 0
        self.w_in, self.w_out = torch.cat(firsts).contiguous(), torch.cat(lasts, dim=1).contiguous()
        self.active = True

    def prepare(self, max_positions):
        if self.active:
            from ..ops.library import joined
            joined()                                       # build or load this part's kernels now, loudly

    def weights(self):
        return [t for t in (self.w_in, self.w_out) if t is not None]

    def apply(self, h, ctx, cache_entry: int, owns_cache: bool):
        """(sum of the sublayers' outputs float32 [T, hidden], None or (rows, weights) still to be added to it)."""
        proj = linear(h, self.w_in, out_dtype=ctx.dtype)
        side = (torch.zeros if self.padded else torch.empty)(h.shape[0], self.w_out.shape[1], dtype=ctx.dtype, device=h.device)
        rows = None
        for m, col, side_col in zip(self.members, self.cols, self.side_cols):
            more = m.fill_side(proj, col, side, side_col, h, ctx, cache_entry, owns_cache)
            if more is not None:
                if rows is not None:
                    raise ValueError("only one sublayer may pass rows on beside its product")
                rows = more
        return linear(side, self.w_out, out_dtype=torch.float32), rows
