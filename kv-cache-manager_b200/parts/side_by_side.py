"""Two mixers that read the same rows, side by side in one layer.

    y = left_scale * left(h) + right_scale * right(h)                                          (``out_norm`` off)
    y = left_scale * w_l * left(h) / rms(left(h)) + right_scale * w_r * right(h) / rms(right(h))        (``out_norm`` on)

rms(v) = sqrt(mean(v^2) + norm_eps) over the model's width, w_l and w_r plain learned vectors [hidden].

At most one of the two keeps paged keys and values.  Each may keep fixed-size state: the call site's state row is then theirs
one behind the other, each part starting at a multiple of four floats.  The sum is not formed here: without ``out_norm`` the two
float32 outputs are returned as (tensor, scale) pairs for the block to hand to the next norm kernel, which adds
them into the stream; with it they are returned as a ``NormedSum``, which the closing norm's kernel forms.

Two staged mixers (see ``parts.base.Mixer``) share launches: their input projections are one product (the matrices are joined
row-wise once, after loading, and the mixers' own parameters become views of the joint one), their heads are prepared by one
launch and gated by one.  In a step of single rows, whose kernels leave most of the device idle, the right mixer's launches
behind the preparation go to a second stream that joins again before the mixers' results are read (``options['branches']``:
'one' keeps to one stream).  ``fuse`` off: each mixer runs by itself.
"""
from __future__ import annotations

import dataclasses

import torch

from ..kernels import library as K
from .base import MIXERS, Mixer, NormedSum, SiteCache, StateSpec, StepContext, run_prepare
from .linear import matmul_nt


_SIDE_STREAMS = {}            # one per device, for all layers


def _up4(n: int) -> int:
    return (n + 3) // 4 * 4


@MIXERS.register("side_by_side")
class SideBySideMixer(Mixer):
    def __init__(self, left: Mixer, right: Mixer, left_scale: float = 1.0, right_scale: float = 1.0, out_norm: bool = False,
                 hidden: int = 0, norm_eps: float = 1e-6, init=("ones_jitter", 0.1)) -> None:
        super().__init__()
        self.left, self.right = self.add_child("left", left), self.add_child("right", right)
        self.left_scale, self.right_scale, self.norm_eps = float(left_scale), float(right_scale), float(norm_eps)
        if left.cache_spec() is not None and right.cache_spec() is not None:
            raise ValueError("side_by_side: both mixers want the call site's cache")
        sizes = []
        for m in (left, right):
            s = m.state_spec()
            if s is not None and (len(s.shape) != 1 or s.dtype != torch.float32):
                raise ValueError("side_by_side: the mixers' states are float32 rows")
            sizes.append(s.shape[0] if s is not None else 0)
        self._state_sizes = tuple(sizes)
        self._state_starts = (0, _up4(sizes[0]))
        self.out_norm = bool(out_norm)
        if self.out_norm:
            self.declare("left_out", (hidden,), init, "vector")
            self.declare("right_out", (hidden,), init, "vector")
        self._multipliers = self._joint = None

    def cache_spec(self):
        return self.left.cache_spec() or self.right.cache_spec()

    def state_spec(self):
        n, (_, at) = self._state_sizes, self._state_starts
        return StateSpec((_up4(at + n[1]),), torch.float32) if any(n) else None

    def prepare(self, device, dtype) -> None:
        left, right = self.left, self.right
        if left.staged and right.staged:
            a, b = left.projection.param("weight"), right.projection.param("weight")
            self._joint = torch.cat([a, b])
            left.projection.set_param("weight", self._joint[:a.shape[0]])
            right.projection.set_param("weight", self._joint[a.shape[0]:])
        super().prepare(device, dtype)
        if self.out_norm:
            self._multipliers = tuple((self.param(n).to(device=device, dtype=torch.float32) * s).contiguous()
                                      for n, s in (("left_out", self.left_scale), ("right_out", self.right_scale)))

    def _sites(self, site: SiteCache):
        """The call site as each mixer sees it: its own part of the state rows."""
        if site.state is None:
            return site, site
        if site.shares is None:
            site.shares = tuple(dataclasses.replace(site, state=site.state[:, at:at + n] if n else None)
                                for at, n in zip(self._state_starts, self._state_sizes))
        return site.shares

    def _two_streams(self, proj: torch.Tensor, mixers, works):
        """Each branch on a stream of its own.  What the side stream's launches read and write is allocated on either stream
        and lives until the join is enqueued; a block freed later is used again on its own stream behind the next fork."""
        main, device = torch.cuda.current_stream(), proj.device
        side = _SIDE_STREAMS.get(device)
        if side is None:
            side = _SIDE_STREAMS[device] = torch.cuda.Stream(device=device)
        outs = [None, None]
        side.wait_stream(main)
        with torch.cuda.stream(side):
            K.gate_heads(proj, [mixers[1].mix(works[1])])
            outs[1] = mixers[1].finish(works[1])
        K.gate_heads(proj, [mixers[0].mix(works[0])])
        outs[0] = mixers[0].finish(works[0])
        main.wait_stream(side)
        return outs

    def forward(self, h: torch.Tensor, ctx: StepContext, site: SiteCache):
        sites, mixers = self._sites(site), (self.left, self.right)
        if self._joint is not None and ctx.options.get("fuse", True):
            proj = matmul_nt(h, self._joint, torch.float32, ctx.options)
            works = [m.begin(proj, at, h.dtype, ctx, s) for m, at, s in zip(mixers, (0, self.left.projection.out_features), sites)]
            run_prepare(proj, works, h.dtype, ctx)
            if ctx.prefill_rows == 0 and ctx.options.get("branches", "two") == "two" and not K.profiling():
                outs = self._two_streams(proj, mixers, works)
            else:
                K.gate_heads(proj, [m.mix(w) for m, w in zip(mixers, works)])
                outs = [m.finish(w) for m, w in zip(mixers, works)]
        else:
            outs = [m.forward(h, ctx, s) for m, s in zip(mixers, sites)]
        if self.out_norm:
            return NormedSum(list(zip(outs, self._multipliers)), self.norm_eps)
        pairs = []
        for y, s in zip(outs, (self.left_scale, self.right_scale)):
            pairs += [(t, c * s) for t, c in y] if isinstance(y, (list, tuple)) else [(y, s)]
        return pairs
