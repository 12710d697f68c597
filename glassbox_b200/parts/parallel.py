"""Two mixers side by side: both read the same input, and the output is left_scale * left + right_scale * right, each side
optionally normed over the model width first (an RMS norm with a gain of its own).

Either mixer may be any registered one; their caches share the layer's cache layer (at most one of them may keep pages, any
may keep a state per request: ``combine_cache_specs``). Each writes its output into a float32 buffer of its own (as under
a wiring that norms a branch: ``ctx.overwrite_output``); one small kernel forms the weighted sum and stores it or adds it
into the residual, in float32. A wiring that norms the branch may take a normed pair over in its parts
(``ctx.accepts_normed_pair`` / ``ctx.normed_pair``) and form the sum on its way over the rows. Where both sides begin with one
stacked product of their input, the two matrices may be one (``shared_projection``): one product then serves both.

The sides do not depend on one another, so the right one runs on the step's second stream where there is one (a fork and a
join in the recorded step), with scratch buffers of its own.
"""
from __future__ import annotations

import torch

from .. import kernels
from ..weights.binding import ParamSpec
from .base import Mixer, build_part, combine_cache_specs, register_part, sub_view
from .linear import linear


class ParallelMixer(Mixer):
    can_overwrite_output = True
    launches_through_kernels_only = False      # (clearing the buffer for a part that adds is a torch operation)

    def __init__(self, spec, *, hidden_size: int):
        super().__init__(spec)
        self.hidden_size = hidden_size
        self.left = build_part("mixer", spec.left, hidden_size=hidden_size)
        self.right = build_part("mixer", spec.right, hidden_size=hidden_size)
        self.left_norm = self.right_norm = None
        if spec.output_norm is not None:
            self.left_norm = build_part("norm", spec.output_norm, hidden_size=hidden_size)
            self.right_norm = build_part("norm", spec.output_norm, hidden_size=hidden_size)
        if spec.shared_projection:
            for part in (self.left, self.right):
                if not part.can_take_projected_input:
                    raise ValueError(f"a mixer of kind {part.spec.kind!r} cannot share its input projection")
                part.projected_input = True
            self.left_cols, self.in_cols = self.left.in_cols, self.left.in_cols + self.right.in_cols

    def sub_parts(self):
        parts = {"left": self.left, "right": self.right}
        if self.left_norm is not None:
            parts.update({"left_norm": self.left_norm, "right_norm": self.right_norm})
        return parts

    def param_specs(self):
        if not self.spec.shared_projection:
            return {}
        return {"w_in": ParamSpec((self.in_cols, self.hidden_size), pieces=self.left.input_pieces() + self.right.input_pieces())}

    def recordable(self, decode_only: bool) -> bool:
        return True

    def cache_spec(self):
        return combine_cache_specs([("left", self.left.cache_spec()), ("right", self.right.cache_spec())])

    def forward(self, ctx, h, residual, cache, writes_cache: bool) -> None:
        n, d = residual.shape
        overwrite = getattr(ctx, "overwrite_output", False)
        takes_pair = getattr(ctx, "accepts_normed_pair", False)
        # what the wiring offers to take over is this mixer's output, not that of either side
        offers = {name: getattr(ctx, name, False) for name in ("accepts_output_bias", "accepts_weighted_rows", "accepts_normed_pair")}
        for name in offers:
            setattr(ctx, name, False)
        inputs = {"left": h, "right": h}
        if self.spec.shared_projection:
            ld = -(-self.in_cols // 4) * 4
            proj = ctx.scratch("parallel_proj", (n, ld), torch.float32)[:, :self.in_cols]
            linear(ctx, h, self.params["w_in"], proj)
            inputs = {"left": proj[:, :self.left_cols], "right": proj[:, self.left_cols:]}
        outs = [ctx.scratch("parallel_" + name, (n, d), torch.float32) for name in ("left", "right")]

        def run(name, part, y):
            ctx.overwrite_output = bool(part.can_overwrite_output)
            if not ctx.overwrite_output:
                y.zero_()
            try:
                part.forward(ctx, inputs[name], y, sub_view(cache, name, part.cache_spec()), writes_cache)
            finally:
                ctx.overwrite_output = overwrite
        side, main = getattr(ctx, "side_stream", None), torch.cuda.current_stream()
        if side is not None and side != main:
            side.wait_stream(main)
            with torch.cuda.stream(side):
                before, ctx.scratch_prefix = ctx.scratch_prefix, ctx.scratch_prefix + "beside_"
                try:
                    run("right", self.right, outs[1])
                finally:
                    ctx.scratch_prefix = before
            run("left", self.left, outs[0])
            main.wait_stream(side)
        else:
            run("left", self.left, outs[0])
            run("right", self.right, outs[1])
        for name, was in offers.items():
            setattr(ctx, name, was)
        s = self.spec
        if self.left_norm is not None:
            lrms, rrms = self.left_norm.as_rms(), self.right_norm.as_rms()
            if overwrite and takes_pair and lrms is not None and rrms is not None and lrms[1] == rrms[1]:
                ctx.normed_pair = kernels.NormedPair(outs[0], outs[1], lrms[0], rrms[0], s.left_scale, s.right_scale, lrms[1])
                return
            for i, norm in enumerate((self.left_norm, self.right_norm)):
                normed = ctx.scratch("parallel_normed_%d" % i, (n, d), torch.float32)
                norm.forward(ctx, outs[i], normed)
                outs[i] = normed
        kernels.scaled_sum(outs[0], outs[1], s.left_scale, s.right_scale, residual, accumulate=not overwrite)


register_part("mixer", "parallel", ParallelMixer, replace=True)
