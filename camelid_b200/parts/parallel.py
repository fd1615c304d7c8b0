"""Several mixers side by side: all read the same rows, and the layer adds the mean of their
outputs, each first RMS-normed over the model width with a weight of its own
(``<prefix><branch>.out``):

    y = (1 / B) * sum over branches b of rmsnorm(mixer_b(x)) * out_b.

A branch is any registered mixer that offers ``branch_output(ctx, x, name)``; each keeps its
own cache or state (the entry's cache needs are the branches' together).

With ``scales`` (a number per branch) the layer's output is the weighted sum of the branches' instead, without norms or
tensors of its own:  y = sum over b of scales[b] * mixer_b(x).  The branches' rows then stand side by side, each times its
scale (``output_rows``, ``scale_output``), and one product with their output matrices side by side makes the sum.
"""
from __future__ import annotations

import torch

from ..csrc import ops
from ..errors import ConfigError
from .base import Part, TensorSpec, build_part, register_part


@register_part("mixer", "parallel")
class ParallelMixers(Part):
    def __init__(self, params, prefix=""):
        super().__init__(params, prefix)
        self.hidden_size = int(params["hidden_size"])
        self.eps = float(params.get("eps", 1e-6))
        self.names = [name for name, _ in params["branches"]]
        self.branches = [build_part("mixer", spec) for _, spec in params["branches"]]
        if not 1 <= len(self.branches) <= 4:
            raise ConfigError("branches", f"1 to 4 mixers can stand side by side, got {len(self.branches)}")
        for name, b in zip(self.names, self.branches):
            if not hasattr(b, "branch_output"):
                raise ConfigError("branches", f"the mixer {b.kind!r} of branch {name!r} cannot stand beside others")
        self.scales = tuple(float(c) for c in params["scales"]) if params.get("scales") is not None else None
        if self.scales is not None:
            if len(self.scales) != len(self.branches):
                raise ConfigError("scales", f"one number per branch: {len(self.branches)} branches, {len(self.scales)} numbers")
            for name, b in zip(self.names, self.branches):
                if not (hasattr(b, "output_rows") and hasattr(b, "scale_output")):
                    raise ConfigError("branches", f"the mixer {b.kind!r} of branch {name!r} cannot enter a weighted sum")
        self.out_w = self.w_joint = None

    @property
    def graph_safe(self):
        return all(b.graph_safe for b in self.branches)

    @property
    def graph_safe_any_step(self):
        return all(b.graph_safe_any_step for b in self.branches)

    def tensor_specs(self):
        specs = {}
        for name, b in zip(self.names, self.branches):
            specs.update(b.tensor_specs())
            if self.scales is None:
                specs[f"{self.prefix}{name}.out"] = TensorSpec((self.hidden_size,), "norm")
        return specs

    def load(self, tensors, device, dtype):
        for b in self.branches:
            b.load(tensors, device, dtype)
        if self.scales is None:
            self.out_w = [tensors[f"{self.prefix}{name}.out"].to(device=device, dtype=torch.float32).contiguous()
                          for name in self.names]
        else:                           # the output matrices' columns side by side; each branch keeps its own as a view
            self.w_joint = torch.cat([b.output_weight() for b in self.branches], dim=1).contiguous()
            at = 0
            for b, c in zip(self.branches, self.scales):
                k = b.output_weight().shape[1]
                b.set_output_weight(self.w_joint[:, at:at + k])
                b.scale_output(c)
                at += k
        # Branches that read the same rows through one stacked input matrix each (``w_in``): all of them stacked
        # once more, so that one product serves every branch; each keeps its rows of it as a view.
        self.w_in = None
        self.in_cols = []
        if len(self.branches) > 1 and all(getattr(b, "w_in", None) is not None for b in self.branches):
            # (each branch's rows padded to a multiple of 8 with zeros: its columns of the product start on 16 bytes)
            padded = [-b.w_in.shape[0] % 8 for b in self.branches]
            pieces = [t for b, pad in zip(self.branches, padded) for t in ([b.w_in, b.w_in.new_zeros((pad, b.w_in.shape[1]))] if pad else [b.w_in])]
            stacked = torch.cat(pieces, dim=0).contiguous()
            at = 0
            for b, pad in zip(self.branches, padded):
                n = b.w_in.shape[0]
                b.w_in = stacked[at:at + n]
                self.in_cols.append((at, n))
                at += n + pad
            self.w_in = stacked

    def cache_spec(self):
        return [b.cache_spec() for b in self.branches]

    def query_tile_sizes(self):
        return [r for b in self.branches for r in b.query_tile_sizes()]

    def workspace_per_row(self):
        return sum(b.workspace_per_row() for b in self.branches)

    def _projections(self, ctx, x):
        """Every branch's columns of the stacked input product (None each where there is no such product): complete rows, or
        split sums on one-token steps where every branch takes those."""
        if self.w_in is None:
            return [None] * len(self.branches)
        from . import linear
        split = ctx.decode and all(getattr(b, "takes_split_rows", False) for b in self.branches)
        proj = (linear.product_f32 if split else linear.product_rows_f32)(ctx, x, self.w_in, "branches_proj")
        return [proj[..., at:at + n] for at, n in self.in_cols]

    def _joint_rows(self, ctx, x):
        rows = ctx.buffer("branches_rows", (ctx.n_rows, self.w_joint.shape[1]))
        at = 0
        for b, proj in zip(self.branches, self._projections(ctx, x)):
            k = b.output_weight().shape[1]
            b.output_rows(ctx, x, rows[:, at:at + k], proj)
            at += k
        return rows

    def forward(self, ctx, x, residual):
        if self.w_joint is not None:
            from . import linear
            linear.add_into_residual(ctx, self._joint_rows(ctx, x), self.w_joint, residual, "o_partial")
            return
        ys = [b.branch_output(ctx, x, f"branch{i}_out", proj) if proj is not None else b.branch_output(ctx, x, f"branch{i}_out")
              for i, (b, proj) in enumerate(zip(self.branches, self._projections(ctx, x)))]
        ops.norm_combine(list(zip(ys, self.out_w)), residual, self.eps, 1.0 / len(self.branches))

    def branch_output(self, ctx, x, name: str):
        """The weighted sum as float32 rows or split sums, for a block that norms it before it is added."""
        from . import linear
        if self.w_joint is None:
            raise ConfigError("branches", "branches whose outputs are normed one by one add into the stream themselves")
        return linear.product_f32(ctx, self._joint_rows(ctx, x), self.w_joint, name)
