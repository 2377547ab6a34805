"""Several mixers side by side on one input, their outputs summed, each normed first or as it is."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds
from ..config.specs import BranchSumSpec, ConfigError
from ..ops import kernels, linear
from ..weights.loader import ParamSpec
from .base import MIXERS, Mixer, SharedProducts, build_part, register_mixer


@register_mixer(BranchSumSpec)
class BranchSum(Mixer):
    """weight * sum_i rmsnorm(branch_i(h)) * w_i.  The branches are ordinary mixers; at most one of them keeps keys and
    values (they share the layer's cache entry), and their states lie one behind the other in the layer's row of the
    state area (each branch is told its ``state_offset``).  The norms of the branches' outputs, their sum and the
    sum into the residual stream are one float32 kernel (csrc/gated_ops.cu).

    Without norms (``out_norms`` None) the result is sum_i scales[i] * branch_i(h).  Branches that can share their products
    (``SharedProducts``) then run as one mixer: one first product for all, one kernel that norms, turns and stores what they need of
    it, each branch's own mixing, one kernel that gates and scales the branches' rows and sets them side by side, and one last product
    over all of them, which adds the branches up (csrc/branch_ops.cu)."""

    takes_out_dtype = True

    def __init__(self, spec: BranchSumSpec, dtype, device):
        super().__init__(spec, dtype, device)
        each = spec.out_norms if spec.out_norms is not None else spec.scales
        if not 1 <= len(spec.branches) <= 4 or each is None or len(each) != len(spec.branches):
            raise ConfigError("a sum of branches takes one to four branches and a norm weight or a factor for each")
        self.branches = [build_part(MIXERS, "mixer", b, dtype, device) for b in spec.branches]
        needs = [b.cache_needs() for b in self.branches]
        if sum(1 for n in needs if n.kv is not None) > 1:
            raise ConfigError("only one branch of a sum may keep keys and values")
        if any(n.state_elems and n.state_dtype != "float32" for n in needs):
            raise ConfigError("branches keep float32 state")
        offset = 0
        for b, n in zip(self.branches, needs):
            if n.state_elems and not hasattr(b, "state_offset"):
                raise ConfigError(f"{type(b).__name__} keeps state but cannot be placed behind another part's (no state_offset)")
            if hasattr(b, "state_offset"):
                b.state_offset = offset
            offset += n.state_elems
        self._needs = CacheNeeds(kv=next((n.kv for n in needs if n.kv is not None), None), state_elems=offset)
        self.out_norms = self.w_in = self.b_in = self.w_o = None
        self.shared = spec.out_norms is None and all(isinstance(b, SharedProducts) and b.can_share() for b in self.branches)
        # the branch that keeps keys and values comes first: its queries must stand at the front of the rows
        self.order = sorted(range(len(self.branches)), key=lambda i: needs[i].kv is None)
        self.columns = []

    def expected_tensors(self):
        out = {}
        for b in self.branches:
            out.update(b.expected_tensors())
        out.update({n: ParamSpec((self.spec.hidden,), init="one_plus_normal") for n in self.spec.out_norms or ()})
        return out

    def take_tensors(self, get):
        for b in self.branches:
            b.take_tensors(get)
        self.out_norms = [get(n) for n in self.spec.out_norms or ()]
        if self.shared:
            ws, bs, os = [], [], []
            for i in self.order:
                w, b = self.branches[i].give_input()
                self.columns.append(sum(t.shape[0] for t in ws))
                ws.append(w)
                bs.append(b)
                os.append(self.branches[i].give_output())
            pad = -sum(t.shape[1] for t in os) % 8           # rows the last product can take with aligned reads
            if pad:
                os.append(os[0].new_zeros(self.spec.hidden, pad))
            self.w_in, self.w_o = torch.cat(ws).contiguous(), torch.cat(os, dim=1).contiguous()
            if any(b is not None for b in bs):
                self.b_in = torch.cat([w.new_zeros(w.shape[0]) if b is None else b.to(w.dtype) for w, b in zip(ws, bs)]).contiguous()

    def prepare(self, max_positions):
        for b in self.branches:
            b.prepare(max_positions)

    def weights(self):
        return ([t for b in self.branches for t in b.weights()] + list(self.out_norms or [])
                + [t for t in (self.w_in, self.b_in, self.w_o) if t is not None])

    def cache_needs(self):
        return self._needs

    def add_normed_to(self, x, norm, scale, ctx, entry, cache_entry, owns_cache) -> bool:
        """x += scale * mixer(norm(x)); branches that can take the norm into their first product."""
        if self.spec.out_norms is None or not all(getattr(b, "takes_out_dtype", False) for b in self.branches):
            return False
        outs = [b.apply(None, ctx, entry, cache_entry, owns_cache, out_dtype=x.dtype, x_norm=(x, norm)) for b in self.branches]
        kernels.normed_sum_add(x, outs, self.out_norms, self.spec.norm_eps, scale * self.spec.weight)
        return True

    def add_scaled_to(self, x, h, scale, ctx, entry, cache_entry, owns_cache) -> None:
        """x += scale * mixer(h) for normed rows h."""
        if self.spec.out_norms is None:
            kernels.scaled_add(x, self.apply(h, ctx, entry, cache_entry, owns_cache, x.dtype).contiguous(), scale)
            return
        outs = [b.apply(h, ctx, entry, cache_entry, owns_cache, **({"out_dtype": x.dtype} if getattr(b, "takes_out_dtype", False) else {}))
                for b in self.branches]
        if len({o.dtype for o in outs}) > 1:
            outs = [o.float() for o in outs]
        kernels.normed_sum_add(x, outs, self.out_norms, self.spec.norm_eps, scale * self.spec.weight)

    def _shared_sum(self, h, ctx, cache_entry, owns_cache, out_dtype):
        proj = linear(h, self.w_in, self.b_in, out_dtype=ctx.dtype)
        runs = [(self.branches[i], col, self.spec.scales[i]) for i, col in zip(self.order, self.columns)]
        jobs = [b.prepare_jobs(proj, col, ctx, cache_entry, owns_cache) for b, col, _ in runs]
        turned = [None] * len(runs)
        normed_at = next((i for i, (n, _) in enumerate(jobs) if n is not None), None)
        turned_at = [i for i, (_, t) in enumerate(jobs) if t is not None]
        if normed_at is not None or turned_at:               # the first job of either kind together, any others after it
            out = kernels.heads_prepare(proj, ctx.tok_pos, ctx.tok_row, None if normed_at is None else jobs[normed_at][0],
                                        jobs[turned_at[0]][1] if turned_at else None)
            if turned_at:
                turned[turned_at[0]] = out
            for i in turned_at[1:]:
                turned[i] = kernels.heads_prepare(proj, ctx.tok_pos, ctx.tok_row, None, jobs[i][1])
        rows = [b.mixed_rows(proj, col, t, ctx, cache_entry, owns_cache) for (b, col, _), t in zip(runs, turned)]
        side = kernels.gate_heads([b.gate_job(r, col, s) for (b, col, s), r in zip(runs, rows)], proj, self.w_o.shape[1])
        return linear(side, self.w_o, out_dtype=out_dtype or ctx.dtype)

    def apply(self, h, ctx, entry, cache_entry, owns_cache, out_dtype=None):
        if self.shared:
            return self._shared_sum(h, ctx, cache_entry, owns_cache, out_dtype)
        y = torch.zeros(h.shape[0], self.spec.hidden, dtype=torch.float32, device=h.device)
        if self.spec.out_norms is None:
            for b, s in zip(self.branches, self.spec.scales):
                wide = {"out_dtype": y.dtype} if getattr(b, "takes_out_dtype", False) else {}
                kernels.scaled_add(y, b.apply(h, ctx, entry, cache_entry, owns_cache, **wide).contiguous(), s)
            return y
        self.add_scaled_to(y, h, 1.0, ctx, entry, cache_entry, owns_cache)
        return y
