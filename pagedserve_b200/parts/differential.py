"""Attention whose heads are the difference of two softmax maps."""

from __future__ import annotations

import torch

from pagedserve_b200.cache.manager import KVNeed
from pagedserve_b200.parts.base import Mixer, register_part
from pagedserve_b200.weights.loader import ParamSpec


@register_part("mixer", "differential_attention")
class DifferentialAttention(Mixer):
    """H query heads on G key/value heads, each with two queries (keys) of ``head_dim`` numbers and one value of ``v_dim``:
    q = W_q x is laid out [head][map][head_dim], k = W_k x likewise.  Every map of every head is divided by its root mean
    square (eps inside the root) and multiplied by a gain of ``head_dim`` numbers, one for all queries and one for all keys;
    queries are then multiplied by 1 + coef ln(floor((p + 1) / every) + 1) of their position p (``q_temp``).  Map i of head h
    is a causal softmax attention a_i over the values of key/value head h / (H / G), scores (q_i . k_i) * scale, and

        o = a_1 - share a_2,    share = exp(lq1 . lk1) - exp(lq2 . lk2) + diff   (one number for the layer)
        o <- o / sqrt(mean(o^2) + eps) * (1 - diff) * sigmoid(W_g x)_h

    The heads are joined and W_o adds the result into the residual row.

    A cached head is [k_1 | k_2] and [v]: the two keys of a head stand side by side in ``slot_dim`` numbers, the larger of
    2 head_dim and v_dim, rounded up to a multiple of 16 in bfloat16.  The two queries of a head become two query heads of
    that size, [q_1 | 0] and [0 | q_2], so every attention kernel runs unchanged, with 2 H query heads on G key/value heads,
    and a group's keys and values are cached and read once for both maps.

    ``kv_source`` False: the layer has no key and value tensors (projections, key gain); its run in the schedule names the
    cache layer of another layer, which has written that step's keys and values before this one runs.

    Launches: the stacked projection (q | k | v | gate), ``diff_prepare`` (norms, factors, cache write), attention,
    ``diff_combine`` (difference, norm, gate), the output product.  Norm statistics, factors, scores, softmax and the
    difference are float32.

    params: hidden_size, n_heads, n_kv_heads, head_dim, v_dim, scale, eps, diff, q_temp (None, or dict(coef, every)),
    kv_source (True), init_std, out_init_std; tensors q, k, v, q.norm, k.norm, lq1, lk1, lq2, lk2, g, o.
    """

    graph_safe = True
    accepts_deferred_norm = True
    takes_result_factor = True

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        p = self.params
        if p["n_heads"] % p["n_kv_heads"]:
            raise ValueError("n_heads must be a multiple of n_kv_heads")
        slot = max(2 * p["head_dim"], p["v_dim"])
        if env.dtype == torch.bfloat16:
            slot = -(-slot // 16) * 16                 # the tensor-core attention kernels take multiples of 16
        if not (0 < slot <= 1024):           # (above 256 the CUDA-core attention kernel runs in bfloat16 too)
            raise ValueError("differential_attention: two keys, or a value, of more than 1024 numbers are not supported")
        self.slot_dim = slot
        self.kv_source = p.get("kv_source", True)
        temp = p.get("q_temp")
        if temp is not None and not (isinstance(temp["every"], int) and temp["every"] > 0):
            raise ValueError("differential_attention: q_temp.every is a positive integer")
        self.q_temp = (float(temp["coef"]), temp["every"]) if temp is not None else None

    def cache_need(self):
        return KVNeed(self.params["n_kv_heads"], self.slot_dim, None)

    def param_specs(self):
        p, std = self.params, self.params.get("init_std", 0.02)
        W, H, G, d, e = p["hidden_size"], p["n_heads"], p["n_kv_heads"], p["head_dim"], p["v_dim"]
        matrix = lambda name, rows, columns=W, s=std: (ParamSpec(self._n(name), (rows, columns), "matmul"), ("normal", s))
        gain = lambda name: (ParamSpec(self._n(name), (d,), "vector"), ("ones_plus_normal", 0.1))
        specs = [matrix("q", 2 * H * d), gain("q.norm")]
        if self.kv_source:
            specs += [matrix("k", 2 * G * d), matrix("v", G * e), gain("k.norm")]
        specs += [(ParamSpec(self._n(name), (d,), "vector"), ("normal", 0.5 * d ** -0.5)) for name in ("lq1", "lk1", "lq2", "lk2")]
        return specs + [matrix("g", H), matrix("o", W, H * e, p.get("out_init_std", std))]

    def bind(self, tensors):
        p = self.params
        t = lambda name: tensors[self._n(name)]
        parts = [t("q")] + ([t("k"), t("v")] if self.kv_source else []) + [t("g")]
        rows = [part.shape[0] for part in parts]
        # every part begins on a multiple of eight columns of the product's rows, and so does the next row
        parts = [piece for part in parts for piece in (part, part.new_zeros((-part.shape[0] % 8, part.shape[1])))]
        self.w_in = torch.cat(parts, dim=0).contiguous()
        starts, at = [], 0
        for count in rows:
            starts.append(at)
            at += -(-count // 8) * 8
        self.k_offset, self.v_offset = (starts[1], starts[2]) if self.kv_source else (0, 0)
        self.gate_offset = starts[-1]
        self.w_o = t("o")
        self.q_gain = t("q.norm").contiguous()
        self.k_gain = t("k.norm").contiguous() if self.kv_source else None
        dot = lambda a, b: torch.dot(t(a).double(), t(b).double())
        self.share = float(torch.exp(dot("lq1", "lk1")) - torch.exp(dot("lq2", "lk2"))) + float(p["diff"])

    def forward(self, x, residual, ctx, layer):
        p, ops, dtype, device = self.params, self.env.ops, self.env.dtype, residual.device
        tokens, H, G, D = x.shape[0], p["n_heads"], p["n_kv_heads"], self.slot_dim
        row = ops.empty((tokens, self.w_in.shape[0]), dtype, device)
        ops.linear(x, self.w_in, None, row)
        queries = ops.empty((tokens, 2 * H * D), dtype, device)
        ops.diff_prepare(row, self.k_offset, self.v_offset, self.q_gain, self.k_gain, float(p["eps"]), self.q_temp, ctx, layer,
                         queries, H, G, p["head_dim"], p["v_dim"], D, has_kv=self.kv_source)
        # (the two maps' results stay float32: their difference may be much smaller than they are)
        maps = ops.empty((tokens, 2 * H * D), torch.float32, device)
        ops.attention(queries, None, None, maps, ctx, layer, 2 * H, G, D, None, float(p["scale"]), write_cache=False)
        context = ops.empty((tokens, H * p["v_dim"]), dtype, device)
        ops.diff_combine(maps, row[:, self.gate_offset:self.gate_offset + H], context, self.share, float(p["eps"]),
                         1.0 - float(p["diff"]), H, p["v_dim"], D)
        ops.linear(context, self.w_o, None, residual, accumulate=True, factor=self.result_factor)
