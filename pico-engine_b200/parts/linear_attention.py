"""Linear attention: a recurrence over a matrix state per head, with a fixed decay per head or a learned one per key channel."""
from __future__ import annotations

import torch

from ..cache import CacheNeeds
from ..config.specs import ConfigError, LinearAttentionSpec, RotaryHalvesSpec, RotaryPairsSpec
from ..ops import kernels, linear
from ..weights.loader import ParamSpec
from .base import Mixer, SharedProducts, first_product, last_product_into, normed_rows, register_mixer


@register_mixer(LinearAttentionSpec)
class LinearAttention(Mixer, SharedProducts):
    """S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; o normed (over all heads together or head by head),
    multiplied by a gate of the mixer's input, projected by W_o.  q, k, v and the gate are one product on concatenated
    weights; activations of q, k, v, the decay (from its logits), the state, the output, its norm and the gate are float32
    in either dtype (csrc/linear_attention.cu, csrc/gated_ops.cu).  The state [heads, head_dim, v_head_dim] is a run of
    the layer's row of the cache's state area, starting at ``state_offset`` (a mixer that holds several mixers places
    them one behind the other).  With a rotation, queries and keys are turned and scaled into float32 rows of their own, which the
    recurrence reads (csrc/branch_ops.cu).  All it reads of the step lies on the device, so a decode step can be a captured graph."""

    takes_out_dtype = True      # apply(..., out_dtype=) gives the product's float32 sums where the caller goes on in float32

    def __init__(self, spec: LinearAttentionSpec, dtype, device):
        super().__init__(spec, dtype, device)
        if (spec.head_decay is None) == (spec.decay_names is None):
            raise ConfigError("linear attention needs either a decay per head or the names of a decay projection")
        if spec.head_decay is not None and len(spec.head_decay) != spec.n_heads:
            raise ConfigError(f"{len(spec.head_decay)} decays for {spec.n_heads} heads")
        if spec.head_dim > 256:
            raise ConfigError(f"head size {spec.head_dim} is not taken: the recurrence kernel takes up to 256")
        if spec.norm_over not in ("heads", "head"):
            raise ConfigError(f"norm_over must be \"heads\" or \"head\", not {spec.norm_over!r}")
        for a in (spec.qk_activation, spec.v_activation):
            if a not in kernels.LA_ACTIVATIONS:
                raise ConfigError(f"activation {a!r} is not known; known: {', '.join(sorted(kernels.LA_ACTIVATIONS))}")
        if spec.gate_activation not in kernels.GATE_ACTIVATIONS:
            raise ConfigError(f"gate activation {spec.gate_activation!r} is not known")
        if spec.position is not None:
            if not isinstance(spec.position, (RotaryPairsSpec, RotaryHalvesSpec)) or getattr(spec.position, "stretch", None) is not None:
                raise ConfigError("linear attention takes rotation of pairs or of halves, not stretched")
            if spec.head_decay is None or spec.qk_activation != "none":
                raise ConfigError("queries and keys are turned where the decay is fixed and they have no activation")
            if spec.position.dims % 2 or spec.position.dims > spec.head_dim:
                raise ConfigError(f"{spec.position.dims} rotated entries do not fit a head of {spec.head_dim}")
        self.freq = None
        self.state_offset = 0
        self.w_in = self.w_o = self.norm = self.head_decay = self.w_a1 = self.w_a2 = self.b_a2 = None

    def _sizes(self):
        s = self.spec
        return s.n_heads * s.head_dim, s.n_heads * s.v_head_dim

    def expected_tensors(self):
        s = self.spec
        qk, vo = self._sizes()
        p = s.prefix
        out = {p + s.q_name: ParamSpec((qk, s.hidden)), p + s.k_name: ParamSpec((qk, s.hidden)),
               p + s.v_name: ParamSpec((vo, s.hidden)), p + s.g_name: ParamSpec((vo, s.hidden)),
               p + s.o_name: ParamSpec((s.hidden, vo))}
        if s.norm_name is not None:
            out[p + s.norm_name] = ParamSpec((vo if s.norm_over == "heads" else s.v_head_dim,), init="one_plus_normal")
        if s.decay_names is not None:
            a1, a2, b = s.decay_names
            out.update({p + a1: ParamSpec((s.decay_rank, s.hidden)), p + a2: ParamSpec((qk, s.decay_rank)), p + b: ParamSpec((qk,))})
        return out

    def take_tensors(self, get):
        s, p = self.spec, self.spec.prefix
        self.w_in = torch.cat([get(p + n) for n in (s.q_name, s.k_name, s.v_name, s.g_name)], dim=0).contiguous()
        self.w_o = get(p + s.o_name)
        self.norm = None if s.norm_name is None else get(p + s.norm_name)
        if s.decay_names is not None:
            a1, a2, b = s.decay_names
            self.w_a1, self.w_a2, self.b_a2 = get(p + a1), get(p + a2), get(p + b)
        else:
            self.head_decay = torch.tensor(s.head_decay, dtype=torch.float32, device=self.device)

    def prepare(self, max_positions):
        from ..ops.library import gated
        gated()                                            # build or load this part's kernels now, loudly
        pos = self.spec.position
        if pos is not None and pos.dims:
            from .attention_gated import halves_frequencies, pair_frequencies
            self.freq = pair_frequencies(pos, self.device) if isinstance(pos, RotaryPairsSpec) else halves_frequencies(pos, self.device)[0]

    def cache_needs(self):
        s = self.spec
        return CacheNeeds(kv=None, state_elems=s.n_heads * s.head_dim * s.v_head_dim)

    def gated_output(self, h, ctx, cache_entry, x_norm=None):
        """norm(o_t) * gate [T, heads * v_head_dim] of the step's tokens; the sequences' states move on.  The input is
        either normed rows ``h`` or ``x_norm`` = (stream, its norm)."""
        s = self.spec
        qk, vo = self._sizes()
        rows = normed_rows(h, x_norm, ctx, self.w_in)
        proj = first_product(*rows, self.w_in, ctx)
        logits = None
        if self.w_a1 is not None:
            if rows[0] is None and not kernels.fused_takes(proj.shape[0], self.w_a1, rows[1]):
                rows = (x_norm[1].forward(x_norm[0], ctx.dtype), None, None, 0.0)
            logits = linear(first_product(*rows, self.w_a1, ctx), self.w_a2, self.b_a2, out_dtype=torch.float32)
        turned = None
        if s.position is not None:
            turned = kernels.heads_prepare(proj, ctx.tok_pos, ctx.tok_row, turned=self.prepare_jobs(proj, 0, ctx, cache_entry, False)[1])
        o = self.mixed_rows(proj, 0, turned, ctx, cache_entry, False, logits)
        return kernels.gated_norm(o, vo if s.norm_over == "heads" else s.v_head_dim, self.norm, s.norm_eps, proj, 2 * qk + vo,
                                  s.gate_activation, ctx.dtype)

    def mixed_rows(self, proj, col, turned, ctx, cache_entry, owns_cache, logits=None):
        s = self.spec
        qk, vo = self._sizes()
        # With a decay per head, prompts run as products of tiles over chunks of 64 tokens; rows that bring a few tokens walk them.
        # With a decay per channel a chunk is walked twice, which pays only where the walk would leave the GPU empty: token after token
        # is a block a (sequence, head, 32 columns of the state).  Measured on a B200 (16 heads of 128 x 128): one prompt of 2,048
        # tokens 319 us in chunks against 709 us, four such prompts 1,985 us against 1,062 us.  (Every way gives the same numbers up to
        # float32 rounding; rows that bring a few tokens, such as the idle rows of a padded step, do not count.)
        if self.head_decay is not None:
            chunked = any(n > 16 for n in ctx.lens)
        else:
            chunked = 0 < sum(1 for n in ctx.lens if n > 64) * s.n_heads * ((s.v_head_dim + 31) // 32) < 192
        # (keys that are scaled but not turned: the scale moves to the queries, the output being linear in either)
        q_scale = s.q_scale if turned is not None else s.q_scale * s.k_scale
        first = 0 if turned is not None else col
        return kernels.linear_attention(proj, first, first + qk, col + 2 * qk, s.n_heads, s.head_dim, s.v_head_dim, ctx.state(cache_entry),
                                        self.state_offset, ctx.row_first, ctx.row_lens, ctx.slots,
                                        chunked=chunked,
                                        head_decay=self.head_decay, decay_logits=logits, inv_tau=1.0 / s.decay_tau,
                                        q_scale=q_scale, qk_activation=s.qk_activation, v_activation=s.v_activation, qk=turned)

    # ---------------------------------------------------------------- beside another mixer on the same input
    def can_share(self):
        return self.w_a1 is None and self.spec.decay_names is None

    def give_input(self):
        w, self.w_in = self.w_in, None
        pad = -w.shape[0] % 8
        return (w if not pad else torch.cat([w, w.new_zeros(pad, w.shape[1])])), None

    def give_output(self):
        w, self.w_o = self.w_o, None
        return w

    def prepare_jobs(self, proj, col, ctx, cache_entry, owns_cache):
        s = self.spec
        if s.position is None:
            return None, None
        return None, kernels.TurnedHeads(s.n_heads, s.head_dim, col, col + s.n_heads * s.head_dim, self.freq,
                                         0 if self.freq is None else s.position.dims, isinstance(s.position, RotaryHalvesSpec), s.k_scale)

    def gate_job(self, rows, col, scale):
        s = self.spec
        qk, vo = self._sizes()
        return kernels.GatedRows(rows, vo if s.norm_over == "heads" else s.v_head_dim, self.norm, s.norm_eps, col + 2 * qk + vo,
                                 s.gate_activation, scale)

    def apply(self, h, ctx, entry, cache_entry, owns_cache, out_dtype=None, x_norm=None):
        return linear(self.gated_output(h, ctx, cache_entry, x_norm), self.w_o, out_dtype=out_dtype or ctx.dtype)

    def add_normed_to(self, x, norm, scale, ctx, entry, cache_entry, owns_cache) -> bool:
        """x += scale * mixer(norm(x)), the norm in the first product and the sum in the last where they take the sizes."""
        last_product_into(x, self.gated_output(None, ctx, cache_entry, (x, norm)), self.w_o, scale, ctx)
        return True
