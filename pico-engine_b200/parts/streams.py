"""A sublayer's place in a residual of several streams."""
from __future__ import annotations

import torch

from ..config.specs import ConfigError, StreamMixSpec
from ..ops import kernels
from ..weights.loader import ParamSpec
from .base import Part


class StreamMix(Part):
    """The weights with which a sublayer reads the streams (``in_weights`` [S]) and with which its output and the old streams make the
    new ones (``out_weights`` [S], ``mix`` [S from, S to]); float32 in either dtype (csrc/branch_ops.cu: one kernel for the entry of one
    sublayer's output and the sum and norm in front of the next)."""

    def __init__(self, spec: StreamMixSpec, dtype, device):
        super().__init__(spec, dtype, device)
        if not 1 <= spec.streams <= kernels.MAX_STREAMS:
            raise ConfigError(f"{spec.streams} streams are not taken: 1 to {kernels.MAX_STREAMS} are")
        self.in_weights = self.out_weights = self.mix = None

    def expected_tensors(self):
        s = self.spec
        return {s.in_name: ParamSpec((s.streams,), init="one_plus_normal"), s.out_name: ParamSpec((s.streams,), init="one_plus_normal"),
                s.mix_name: ParamSpec((s.streams, s.streams), init="identity_plus_normal")}

    def take_tensors(self, get):
        s = self.spec
        self.in_weights, self.out_weights, self.mix = (get(n).to(torch.float32).contiguous() for n in (s.in_name, s.out_name, s.mix_name))

    def prepare(self, max_positions):
        from ..ops.library import gated
        gated()                                            # build or load this part's kernels now, loudly
