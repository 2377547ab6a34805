"""Grouped softmax attention whose heads are the normed difference of two maps over the same values."""
from __future__ import annotations

import math

import torch

from ..cache import CacheNeeds, KVNeed
from ..config.specs import ConfigError, DifferentialAttentionSpec, NoPositionSpec, RotaryHalvesSpec
from ..ops import kernels, linear
from ..weights.loader import ParamSpec
from .attention_gated import halves_frequencies
from .base import JoinedProducts, Mixer, register_mixer


@register_mixer(DifferentialAttentionSpec)
class DifferentialAttention(Mixer, JoinedProducts):
    """One product for q, k and v; norm of every map's query and key rows, rotation and cache write in one kernel; attention over the cache
    with the two maps' difference, its norm and scale (csrc/attention_diff*.cu, csrc/joined_ops.cu); the output projection.

    The rows of W_q are put into the order [key/value head][map][head of the group] when they are loaded, so that the heads of a group that
    share a map's keys are neighbours; the cache keeps two key heads (one a map) and one value head per key/value head.  Norms, angles,
    scores, softmax, lambda and the difference with its norm are float32 in either dtype."""

    takes_out_dtype = True

    def __init__(self, spec: DifferentialAttentionSpec, dtype, device):
        super().__init__(spec, dtype, device)
        if spec.n_heads % spec.n_kv_heads:
            raise ConfigError(f"{spec.n_heads} query heads cannot share {spec.n_kv_heads} key/value heads evenly")
        pos = spec.position
        if not isinstance(pos, (NoPositionSpec, RotaryHalvesSpec)) or getattr(pos, "stretch", None) is not None:
            raise ConfigError("differential attention takes rotation of halves (by bands, not by a ramp) or no position encoding")
        self.rot_dims = pos.dims if isinstance(pos, RotaryHalvesSpec) else 0
        if self.rot_dims % 2 or self.rot_dims > spec.head_dim:
            raise ConfigError(f"{self.rot_dims} rotated entries do not fit a head of {spec.head_dim}")
        if spec.head_dim > 256 or spec.v_head_dim > 256:
            raise ConfigError(f"head sizes {spec.head_dim}/{spec.v_head_dim} are not taken: up to 256 are")
        if spec.window is not None and spec.window <= 0:
            raise ConfigError(f"window {spec.window} must be positive")
        if len(spec.lambda_names) != 4:
            raise ConfigError("lambda is made of four vectors")
        self.w_in = self.w_o = self.q_norm = self.k_norm = self.freq = None
        self.lam = 0.0

    def _widths(self):
        s = self.spec
        return 2 * s.n_heads * s.head_dim, 2 * s.n_kv_heads * s.head_dim, s.n_kv_heads * s.v_head_dim, s.n_heads * s.v_head_dim

    def expected_tensors(self):
        s, p = self.spec, self.spec.prefix
        q, k, v, o = self._widths()
        out = {p + s.q_name: ParamSpec((q, s.hidden)), p + s.k_name: ParamSpec((k, s.hidden)), p + s.v_name: ParamSpec((v, s.hidden)),
               p + s.o_name: ParamSpec((s.hidden, o))}
        out.update({p + n: ParamSpec((s.head_dim,), init="one_plus_normal") for n in (s.q_norm, s.k_norm) if n is not None})
        out.update({p + n: ParamSpec((s.head_dim,), init="normal") for n in s.lambda_names})
        return out

    def take_tensors(self, get):
        s, p = self.spec, self.spec.prefix
        G, per = s.n_kv_heads, s.n_heads // s.n_kv_heads
        q = get(p + s.q_name).view(G, per, 2, s.head_dim, s.hidden).transpose(1, 2).reshape(-1, s.hidden)
        parts = [q, get(p + s.k_name), get(p + s.v_name)]
        pad = -sum(t.shape[0] for t in parts) % 8          # rows of the product stay aligned for the attention kernels' vector loads
        if pad:
            parts.append(parts[0].new_zeros(pad, s.hidden))
        self.w_in, self.w_o = torch.cat(parts, dim=0).contiguous(), get(p + s.o_name)
        self.q_norm, self.k_norm = (None if n is None else get(p + n) for n in (s.q_norm, s.k_norm))
        l1, l2, l3, l4 = (get(p + n).double() for n in s.lambda_names)
        self.lam = 0.0 if self.device == "meta" or l1.is_meta else math.exp(float((l1 * l2).sum())) - math.exp(float((l3 * l4).sum())) + s.lambda_base

    def prepare(self, max_positions):
        from ..ops.library import joined, mixers
        joined(), mixers()                                 # build or load this part's kernels now, loudly
        if self.rot_dims:
            self.freq, _ = halves_frequencies(self.spec.position, self.device)

    def weights(self):
        return [t for t in (self.w_in, self.w_o, self.q_norm, self.k_norm) if t is not None]

    def cache_needs(self):
        s = self.spec
        return CacheNeeds(kv=KVNeed(2 * s.n_kv_heads, s.head_dim, s.window, v_head_dim=s.v_head_dim, v_heads=s.n_kv_heads))

    def _heads_into(self, proj, side, side_col, ctx, cache_entry, owns_cache):
        """The heads' outputs into columns ``side_col`` .. of side, from the first product's rows (whose queries stand at the front)."""
        s, kv = self.spec, ctx.kv(cache_entry)
        if not owns_cache:
            raise ConfigError("differential attention writes keys and values of its own")
        kernels.heads_norm_store(proj, 2 * s.n_heads, 2 * s.n_kv_heads, s.n_kv_heads, s.head_dim, s.v_head_dim, self.q_norm, self.k_norm, s.norm_eps,
                                 self.freq, self.rot_dims, ctx.tok_pos, ctx.tok_row, kv.k, kv.v, kv.table, kv.stride)
        kernels.attention_maps(proj, s.n_heads, s.n_kv_heads, s.head_dim, s.v_head_dim, kv.k, kv.v, kv.table, kv.stride, ctx.tok_pos, ctx.tok_row,
                               s.window, s.scale, self.lam, s.norm_eps, s.out_scale, side, side_col, ctx)

    def apply(self, h, ctx, entry, cache_entry, owns_cache, out_dtype=None):
        proj = linear(h, self.w_in, out_dtype=ctx.dtype)
        heads = torch.empty(h.shape[0], self._widths()[3], dtype=ctx.dtype, device=h.device)
        self._heads_into(proj, heads, 0, ctx, cache_entry, owns_cache)
        return linear(heads, self.w_o, out_dtype=out_dtype or ctx.dtype)

    # ---------------------------------------------------------------- beside another sublayer on the same rows
    def can_join(self):
        return True

    def lend_products(self):
        w = self.w_in, self.w_o
        self.w_in = self.w_o = None
        return w

    def fill_side(self, proj, col, side, side_col, h, ctx, cache_entry=None, owns_cache=True):
        if col:
            raise ConfigError("an attention's queries stand at the front of the rows")
        self._heads_into(proj, side, side_col, ctx, cache_entry, owns_cache)
