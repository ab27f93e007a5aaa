"""Gated linear attention: a linear recurrence whose matrix state decays per key channel by a gate of the token."""

from __future__ import annotations

import torch

from pagedserve_b200.cache.manager import StateNeed
from pagedserve_b200.parts.base import Mixer, register_part
from pagedserve_b200.weights.loader import ParamSpec


@register_part("mixer", "gated_linear_attention")
class GatedLinearAttention(Mixer):
    """q = W_q x * dim^(-1/2), k = W_k x (heads x dim), v = W_v x (heads x v_dim); the decay of every head and key channel
    is alpha = sigmoid(z)^(1 / tau), z = W_a2 (W_a1 x) + b, a number in (0, 1).  Per head, with S a dim x v_dim matrix that
    starts at zero:

        S[i, j] <- alpha[i] S[i, j] + k[i] v[j],        o[j] = sum_i q[i] S[i, j]

    Each head's o is divided by its root mean square and multiplied by a gain of v_dim numbers (one for all heads), the
    heads are joined, multiplied by silu(W_g x), and W_o adds the result into the residual row.

    A request keeps S (float32) in its slot: a prompt portion runs its tokens in order from the stored state and leaves the
    new one there, a decode step is a portion of one token.  The projections (W_a1's too) are one product in
    the compute type; everything behind it, from the decay's argument on, is float32 (csrc/gla.cu).

    params: hidden_size, n_heads, head_dim, v_dim, tau, eps, random_decay_rank (the inner size of W_a1 / W_a2, which only a
    file gives, for random weights), init_std, out_init_std; tensors q, k, v, g, o, norm, a1, a2, a2.b.
    """

    graph_safe = True
    accepts_deferred_norm = True
    scales_joint = True

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        p = self.params
        if not p["tau"] > 0:
            raise ValueError("gated_linear_attention: tau must be positive")
        self.k_width = p["n_heads"] * p["head_dim"]
        self.v_width = p["n_heads"] * p["v_dim"]

    def state_need(self):
        p = self.params
        return StateNeed((p["n_heads"] * p["head_dim"] * p["v_dim"],), "float32")

    def param_specs(self):
        p = self.params
        W, rank, std = p["hidden_size"], p.get("random_decay_rank", 16), p.get("init_std", 0.02)
        return [(ParamSpec(self._n("q"), (self.k_width, W), "matmul"), ("normal", std)),
                (ParamSpec(self._n("k"), (self.k_width, W), "matmul"), ("normal", std)),
                (ParamSpec(self._n("v"), (self.v_width, W), "matmul"), ("normal", std)),
                (ParamSpec(self._n("g"), (self.v_width, W), "matmul"), ("normal", std)),
                (ParamSpec(self._n("a1"), (-1, W), "matmul"), ("normal", std, (rank, W))),
                (ParamSpec(self._n("a2"), (self.k_width, -1), "vector"), ("normal", rank ** -0.5, (self.k_width, rank))),
                (ParamSpec(self._n("a2.b"), (self.k_width,), "vector"), ("normal", 1.0)),
                (ParamSpec(self._n("norm"), (p["v_dim"],), "vector"), ("ones_plus_normal", 0.1)),
                (ParamSpec(self._n("o"), (W, self.v_width), "matmul"), ("normal", p.get("out_init_std", std)))]

    def bind(self, tensors):
        t = lambda name: tensors[self._n(name)]
        a1, self.a2 = t("a1"), t("a2").contiguous()
        rank = a1.shape[0]
        if rank == 0 or self.a2.shape[1] != rank:
            raise ValueError("gated_linear_attention: the two matrices of the decay do not fit each other")
        # a row of the product ends on a multiple of eight numbers: rows of zeros behind the decay's
        pad = -(2 * self.k_width + 2 * self.v_width + rank) % 8
        self.w_in = torch.cat([t("q"), t("k"), t("v"), t("g"), a1, a1.new_zeros((pad, a1.shape[1]))], dim=0).contiguous()
        self.offsets = (0, self.k_width, 2 * self.k_width, 2 * self.k_width + self.v_width,
                        2 * (self.k_width + self.v_width))
        self.bias, self.gain = t("a2.b").contiguous(), t("norm").contiguous()
        self.w_o = t("o")

    def joint_in(self):
        return self.w_in, None

    def joint_out(self):
        return self.w_o, None

    def joint_mix(self, projected, context, ctx, layer, factor=1.0):
        p = self.params
        self.env.ops.gla_recurrence(projected, self.offsets, self.a2, self.bias, p["tau"], p["head_dim"] ** -0.5, self.gain,
                                    p["eps"], factor, layer.state, ctx, context, p["n_heads"], p["head_dim"], p["v_dim"])

    def forward(self, x, residual, ctx, layer):
        ops = self.env.ops
        projected = ops.empty((x.shape[0], self.w_in.shape[0]), self.env.dtype, residual.device)
        ops.linear(x, self.w_in, None, projected)
        context = ops.empty((x.shape[0], self.v_width), self.env.dtype, residual.device)
        self.joint_mix(projected, context, ctx, layer)
        ops.linear(context, self.w_o, None, residual, accumulate=True)
