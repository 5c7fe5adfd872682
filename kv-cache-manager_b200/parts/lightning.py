"""Lightning attention: a linear-attention mixer with a fixed-size state per request and ONE constant decay per head.

Per head a float32 matrix S [dk, dv], zero at a request's start, is carried from token to token:

    S <- decay_h S + k v^T;    o = S^T q

with q = silu(W_q h), k = silu(W_k h) (heads x dk) and v = silu(W_v h) (heads x dv); no other scale.  The heads' outputs
side by side are divided by their root mean square over all of them and multiplied by a weight [heads * dv] and
by sigmoid(W_g h), and go through the output projection.

State of a request: one float32 row per call site, S of every head.  One product gives q | k | v | g (float32 result).
The recurrence is the engine's matrix-state scan in its linear form (csrc/cuda/delta_rule.cu) with the same decays for
every row; it applies SiLU to q, k and v as it stages them.  With bfloat16 storage the portions of more than a few
tokens take the chunked form on the tensor cores instead (csrc/cuda/linear_chunk.cu; ``options['scan']``: 'tokens' forces
the token-by-token kernel, 'chunks' the chunked one).  Everything between the two products is float32 in both storage
dtypes, but for the chunked form's q, k and v, which are bfloat16 operands.
"""
from __future__ import annotations

from typing import Sequence

import torch

from ..kernels import library as K
from .base import MIXERS, Mixer, SiteCache, StateSpec, StepContext
from .linear import Linear


CHUNKED_MIN_TOKENS = 32       # portions at least this long take the chunked form


def takes_chunks(ctx: StepContext, storage: torch.dtype, dk: int) -> bool:
    """Whether a step's portions take the chunked form (its single rows never do)."""
    mode = ctx.options.get("scan", "auto")
    return (mode == "chunks" or (mode == "auto" and storage == torch.bfloat16 and ctx.max_q_len >= CHUNKED_MIN_TOKENS)) \
        and ctx.prefill_tiles > 0 and K.linear_chunk_supported(dk)


def constant_decay_recurrence(proj: torch.Tensor, bases, decay: torch.Tensor, state: torch.Tensor, ctx: StepContext, o: torch.Tensor,
                              heads: int, dk: int, dv: int, storage: torch.dtype, silu: bool = False, exact: bool = False, **turn) -> None:
    """S <- decay_h S + k v^T; o = S^T q over the step's rows, from and into ``state``; ``decay`` float32 [1, heads], q, k and v at
    ``bases`` of the float32 rows ``proj``.  16-bit storage: portions of CHUNKED_MIN_TOKENS and more in chunks on the tensor
    cores (``exact``: with queries and keys in two parts each; ``turn``: the chunked kernel's own rotation of their rows)."""
    rows = decay.expand(proj.shape[0], heads)
    if takes_chunks(ctx, storage, dk):
        if ctx.decode_seqs:                                                          # the single-row entries come first
            K.state_scan(K.SCAN_LINEAR, proj, bases, None, rows, None, state, ctx, o, heads, heads, dk, dv, silu=silu, seqs=ctx.decode_seqs)
        K.linear_chunk(proj, bases, decay, state, ctx, o, heads, heads, dk, dv, silu=silu, exact=exact, **turn)
    else:
        K.state_scan(K.SCAN_LINEAR, proj, bases, None, rows, None, state, ctx, o, heads, heads, dk, dv, silu=silu)


@MIXERS.register("lightning")
class LightningAttention(Mixer):
    def __init__(self, hidden: int, heads: int, dk: int, dv: int, decay: Sequence[float], norm_eps: float) -> None:
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"lightning: {len(decay)} decays for {heads} heads")
        self.hidden, self.heads, self.dk, self.dv, self.norm_eps = hidden, heads, dk, dv, float(norm_eps)
        self.decay = tuple(float(d) for d in decay)
        n = heads * dv
        self.qkvg = self.add_child("qkvg", Linear(hidden, heads * 2 * dk + 2 * n, hidden ** -0.5))
        self.o = self.add_child("o", Linear(n, hidden, n ** -0.5))
        self.declare("norm", (n,), ("ones_jitter", 0.1), "vector")
        self._norm = self._decay = None

    def state_spec(self) -> StateSpec:
        return StateSpec((self.heads * self.dk * self.dv,), torch.float32)

    def prepare(self, device, dtype) -> None:
        super().prepare(device, dtype)
        if self.dk > K.delta_scan_max_dk():
            raise ValueError(f"lightning: key size {self.dk} exceeds the recurrence kernel's {K.delta_scan_max_dk()}")
        self._norm = self.param("norm").to(device=device, dtype=torch.float32).contiguous()
        self._decay = torch.tensor(self.decay, dtype=torch.float32, device=device).view(1, self.heads)

    def forward(self, h: torch.Tensor, ctx: StepContext, site: SiteCache) -> torch.Tensor:
        T, H, dk, dv = h.shape[0], self.heads, self.dk, self.dv
        n, v0 = H * dv, 2 * H * dk
        proj = self.qkvg.forward(h, ctx, out_dtype=torch.float32)
        o = torch.empty((T, n), dtype=torch.float32, device=h.device)                # (the scan zeroes padding rows)
        constant_decay_recurrence(proj, (0, H * dk, v0), self._decay, site.state, ctx, o, H, dk, dv, h.dtype, silu=True)
        gated = torch.empty((T, n), dtype=h.dtype, device=h.device)
        K.group_rms_gate(o, proj[:, v0 + n:], self._norm, gated, n, self.norm_eps, False, "sigmoid")
        return self.o.forward(gated, ctx, out_dtype=torch.float32)
