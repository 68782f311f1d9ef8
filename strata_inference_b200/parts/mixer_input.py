"""Parts between a layer's first norm and its mixer ("mixer_input").

``short_conv``: x <- x + conv(x), a causal convolution over time on each channel of the normed
rows, without a bias.  Parameter ``taps`` n: conv(x)_t = sum_j weight[:, j] x_(t - n + 1 + j), zeros
before the sequence's start.  The last n - 1 normed rows of a sequence are state of their own
(``CacheNeed.inputs``, 32-bit) in every schedule position, whatever the mixer keeps beside it.
Sums are 32-bit (csrc/short_conv.cu).

Steps of one bfloat16 row per sequence between RMS norms take the residual step ahead of the
mixer ("norm of the sub-layer's output, add, norm") and the convolution as one launch
(``add_norm``).
"""

from __future__ import annotations

from typing import Dict, Mapping, Optional

import torch

from ..cache.paged import StateNeed
from ..config.spec import ConfigError
from ..kernels import native
from ..weights.arena import Piece, Resident
from ..weights.loader import TensorDecl
from .registry import register_mixer_input


class ShortConv:
    captures_prompts = True      # sequences, slots and counts are read on the device only

    @staticmethod
    def tensors(params: Mapping, hidden: int) -> Dict[str, TensorDecl]:
        return {"weight": TensorDecl((hidden, int(params["taps"])), init="norm")}

    @staticmethod
    def resident(params: Mapping, hidden: int) -> Dict[str, Resident]:
        return {"weight": Resident((hidden, int(params["taps"])), torch.float32, (Piece("weight"),))}

    def __init__(self, params: Mapping, hidden: int, weights: Mapping[str, torch.Tensor], rt):
        self.rt = rt
        self.hidden = hidden
        self.taps = int(params["taps"])
        if not 1 <= self.taps <= 64:
            raise ConfigError(f"short_conv: {self.taps} taps (1 to 64)")
        # (neighbouring threads take neighbouring channels: tap by tap)
        self.w = weights["weight"].t().contiguous()

    def state_need(self) -> Optional[StateNeed]:
        # (whole groups of 4 floats, so that every slot's state begins on a 16-byte boundary)
        return StateNeed((-(-(self.taps - 1) * self.hidden // 4) * 4,)) if self.taps > 1 else None

    def _state(self, ctx, entry: int) -> Optional[torch.Tensor]:
        return ctx.input_state(entry) if self.taps > 1 else None

    def forward(self, x: torch.Tensor, ctx, entry: int) -> torch.Tensor:
        return native.short_conv(x, torch.empty_like(x), self.w, self._state(ctx, entry), ctx)

    def fused_with_norm(self, ctx) -> bool:
        """Whether this step's residual add and norms may run together with the convolution."""
        return (self.rt.dtype == torch.bfloat16 and ctx.max_count == 1 and ctx.n_rows == ctx.n_seqs
                and native.add_norm_conv_supports(self.hidden))

    def add_norm(self, y: torch.Tensor, post, h: torch.Tensor, nxt, ctx, entry: int) -> torch.Tensor:
        """h += post(y) (or y); returns x + conv(x) with x = nxt(h); ``post`` and ``nxt`` RMS norms."""
        return native.add_norm_conv(y, post.gain if post is not None else None, post.eps if post is not None else 0.0,
                                    h, nxt.gain, nxt.eps, self.w, self._state(ctx, entry), torch.empty_like(y), ctx)


register_mixer_input("short_conv", ShortConv)
