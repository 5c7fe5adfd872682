"""Retention: linear attention with a fixed-size state per request, a fixed decay per head and rotated queries and keys.

Per head a float32 matrix S [dk, dv], zero at a request's start, is carried from token to token:

    S <- decay_h S + k v^T;    o = S^T q

with q = rot(W_q h), k = rot(W_k h) * dk^-1/2 (heads x dk; the rotation is the ``position`` part's) and v = W_v h (heads x dv).
Each head's o is divided by its root mean square over dv (no weight), the heads side by side are multiplied by SiLU(W_g h)
and go through the output projection.

State of a request: one float32 row per call site, S of every head.  A staged mixer (see ``parts.base.Mixer``): one product gives
q | k | v | g (float32), one launch turns and scales q and k in place (the chunked recurrence turns its rows itself, as it
reads them), the recurrence is that of ``parts.lightning``, one launch normalises and gates.  Everything between the two products is float32 in both storage dtypes; in the chunked form
of the recurrence v is a bfloat16 operand (a plain projection), q and k are split in two bfloat16 parts.
"""
from __future__ import annotations

from typing import Sequence

import torch

from ..kernels import library as K
from .base import MIXERS, Mixer, PositionEncoding, SiteCache, StagedWork, StateSpec, StepContext
from .lightning import constant_decay_recurrence, takes_chunks
from .linear import Linear
from .rope import STEP_TABLE_ROWS


@MIXERS.register("retention")
class Retention(Mixer):
    staged = True

    def __init__(self, hidden: int, heads: int, dk: int, dv: int, decay: Sequence[float], position: PositionEncoding, norm_eps: float) -> None:
        super().__init__()
        if len(decay) != heads:
            raise ValueError(f"retention: {len(decay)} decays for {heads} heads")
        if getattr(position, "rotary_dim", 0) > dk:
            raise ValueError("retention: the rotation covers at most the head's own size")
        self.hidden, self.heads, self.dk, self.dv, self.norm_eps = hidden, heads, dk, dv, float(norm_eps)
        self.decay = tuple(float(d) for d in decay)
        self.position = self.add_child("position", position)
        self.qkvg = self.add_child("qkvg", Linear(hidden, 2 * heads * (dk + dv), hidden ** -0.5))
        self.o = self.add_child("o", Linear(heads * dv, hidden, (heads * dv) ** -0.5))
        self._decay = None

    @property
    def projection(self) -> Linear:
        return self.qkvg

    def state_spec(self) -> StateSpec:
        return StateSpec((self.heads * self.dk * self.dv,), torch.float32)

    def prepare(self, device, dtype) -> None:
        super().prepare(device, dtype)
        if self.dk > K.delta_scan_max_dk():
            raise ValueError(f"retention: key size {self.dk} exceeds the recurrence kernel's {K.delta_scan_max_dk()}")
        self._decay = torch.tensor(self.decay, dtype=torch.float32, device=device).view(1, self.heads)

    def begin(self, proj: torch.Tensor, base: int, dtype: torch.dtype, ctx: StepContext, site: SiteCache) -> StagedWork:
        work, pos, n = StagedWork(proj, base, dtype, ctx, site), self.position, self.heads * self.dk
        rows, table, work.turn = ctx.rows, None, {}
        if pos.inv_freq is not None and ctx.prefill_rows >= STEP_TABLE_ROWS:
            table = pos.step_table(ctx)
            if takes_chunks(ctx, dtype, self.dk) and not pos.interleaved and ctx.options.get("fuse", True) \
                    and K.linear_chunk_turns(proj.shape[1], (base, base + n, base + 2 * n), self.dk, self.dv, pos.rotary_dim // 2):
                work.turn = dict(table=table, amplitude=pos.amplitude, k_scale=self.dk ** -0.5)
                rows = ctx.decode_seqs                      # the portions' rows are turned where they are read
        turn = dict(inv_freq=pos.inv_freq, amplitude=pos.amplitude, interleaved=pos.interleaved, table=table, rows=rows)
        if pos.inv_freq is not None and rows:
            work.segments.append(K.HeadSegment(self.heads, self.dk, base, "float", proj, out_col=base, **turn))
        if rows:
            work.segments.append(K.HeadSegment(self.heads, self.dk, base + n, "float", proj, out_col=base + n, scale=self.dk ** -0.5, **turn))
        return work

    def mix(self, work: StagedWork) -> K.GateSegment:
        T, n, nk, base = work.proj.shape[0], self.heads * self.dv, self.heads * self.dk, work.base
        o = torch.empty((T, n), dtype=torch.float32, device=work.proj.device)        # (the recurrence zeroes padding rows)
        constant_decay_recurrence(work.proj, (base, base + nk, base + 2 * nk), self._decay, work.site.state, work.ctx, o, self.heads,
                                  self.dk, self.dv, work.dtype, exact=True, **work.turn)
        work.out = torch.empty((T, n), dtype=work.dtype, device=work.proj.device)
        return K.GateSegment(o, work.out, self.heads, self.dv, base + 2 * nk + n, self.norm_eps, "silu")

    def finish(self, work: StagedWork) -> torch.Tensor:
        return self.o.forward(work.out, work.ctx, out_dtype=torch.float32)

    def forward(self, h: torch.Tensor, ctx: StepContext, site: SiteCache) -> torch.Tensor:
        return self.forward_staged(h, ctx, site)
