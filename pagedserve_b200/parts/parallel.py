"""Mixers side by side."""

from __future__ import annotations

import dataclasses

import torch

from pagedserve_b200.cache.manager import StateNeed
from pagedserve_b200.parts.base import Mixer, create_part, register_part


def padded(count: int) -> int:
    """State of one owner begins on a multiple of four numbers (16 bytes)."""
    return -(-count // 4) * 4


def state_share(layer, first: int, count: int):
    """``layer`` with the numbers [first, first + count) of every slot's state as its state."""
    return dataclasses.replace(layer, state=layer.state[:, first:first + count])


@register_part("mixer", "parallel")
class ParallelMixers(Mixer):
    """sum_i scale_i * mixer_i(x): several mixers read the same row.  Their projections are one product over the stacked
    matrices, their results stand side by side in one row, and one product over the joined output matrices adds the sum
    up (biases of the output projections, times their mixer's scale, included).

    The scales are not rounded into matrices: a mixer that can (``scales_joint``) multiplies its result by its scale over
    the common one in float32, and the common one, that of the mixer that cannot, is left to the block
    (``output_scale``).

    params: hidden_size, mixers: a list of (kind, params, prefix, scale); at most one of them keeps keys and values in
    pages, and at most one cannot scale its result."""

    graph_safe = True
    accepts_deferred_norm = True

    def __init__(self, params, prefix, env):
        from pagedserve_b200.models.spec import PartSpec

        super().__init__(params, prefix, env)
        self.members, self.scales = [], []
        for kind, values, inner_prefix, scale in self.params["mixers"]:
            self.members.append(create_part("mixer", PartSpec(kind, values, prefix + inner_prefix), env))
            self.scales.append(float(scale))
        if not all(member.graph_safe for member in self.members):
            self.graph_safe = False
        if sum(member.cache_need() is not None for member in self.members) > 1:
            raise ValueError("parallel: more than one mixer with keys and values in pages")
        fixed = [scale for member, scale in zip(self.members, self.scales) if not member.scales_joint]
        if len(fixed) > 1:
            raise ValueError("parallel: more than one mixer that cannot scale its result")
        # (a scale of zero takes its mixer out: its columns of the output matrix become zeros)
        self.output_scale = fixed[0] if fixed and fixed[0] != 0.0 else 1.0

    def cache_need(self):
        return next((need for need in (member.cache_need() for member in self.members) if need is not None), None)

    def _state_counts(self):
        counts = []
        for member in self.members:
            need = member.state_need()
            if need is not None and (need.dtype != "float32" or len(need.shape) != 1):
                raise ValueError("parallel: state is rows of float32 numbers")
            counts.append(need.shape[0] if need is not None else 0)
        return counts

    def state_need(self):
        total = sum(padded(count) for count in self._state_counts())
        return StateNeed((total,), "float32") if total else None

    def param_specs(self):
        return [spec for member in self.members for spec in member.param_specs()]

    def bind(self, tensors):
        matrices, biases, out_matrices = [], [], []
        self.in_columns, self.out_columns = [], []
        self.b_out = None
        first = column = 0
        for member, scale in zip(self.members, self.scales):
            member.bind(tensors)
            w, b = member.joint_in()
            pad = -w.shape[0] % 8                            # the next mixer's columns begin on a multiple of eight
            matrices += [w, w.new_zeros((pad, w.shape[1]))]
            b = torch.zeros(w.shape[0], dtype=torch.float32, device=w.device) if b is None else b
            biases += [b, b.new_zeros(pad)]
            self.in_columns.append((first, w.shape[0]))
            first += w.shape[0] + pad
            w_o, b_o = member.joint_out()
            pad = -w_o.shape[1] % 8
            if scale == 0.0 and not member.scales_joint:
                w_o = torch.zeros_like(w_o)
            out_matrices += [w_o, w_o.new_zeros((w_o.shape[0], pad))]
            self.out_columns.append((column, w_o.shape[1], pad))
            column += w_o.shape[1] + pad
            if b_o is not None:
                b_o = b_o * (scale / self.output_scale)      # float32
                self.b_out = b_o if self.b_out is None else self.b_out + b_o
        self.w_in = torch.cat(matrices, dim=0).contiguous()
        self.b_in = torch.cat(biases).contiguous()
        self.w_out = torch.cat(out_matrices, dim=1).contiguous()

    def forward(self, x, residual, ctx, layer):
        ops = self.env.ops
        projected = ops.empty((x.shape[0], self.w_in.shape[0]), self.env.dtype, residual.device)
        ops.linear(x, self.w_in, self.b_in, projected)
        context = ops.empty((x.shape[0], self.w_out.shape[1]), self.env.dtype, residual.device)
        at = 0
        counts = self._state_counts()
        for index, member in enumerate(self.members):
            first, rows = self.in_columns[index]
            column, width, pad = self.out_columns[index]
            own = layer
            if layer.state is not None:
                own = state_share(layer, at, counts[index])
                at += padded(counts[index])
            factor = self.scales[index] / self.output_scale if member.scales_joint else 1.0
            member.joint_mix(projected[:, first:first + rows], context[:, column:column + width], ctx, own, factor=factor)
            if pad:
                context[:, column + width:column + width + pad].zero_()
        ops.linear(context, self.w_out, self.b_out, residual, accumulate=True)
