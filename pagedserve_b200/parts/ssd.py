"""State-space mixer: a matrix state per head that shrinks by one number per token (Mamba-2)."""

from __future__ import annotations

import torch

from pagedserve_b200.cache.manager import StateNeed
from pagedserve_b200.parts.base import Mixer, register_part
from pagedserve_b200.parts.norms import DeferredNorm, LayerNorm
from pagedserve_b200.parts.parallel import padded, state_share
from pagedserve_b200.weights.loader import ParamSpec


@register_part("mixer", "state_space")
class StateSpaceMixer(Mixer):
    """One projection makes z | x | B | C | dt of a token (H heads of P numbers each for z and x, G groups of N numbers for B
    and C, one number per head for dt).  x, B and C pass a causal convolution over time, channel by channel, with a bias and
    silu; then per head h, with the B and C of group h / (H / G) and S an N x P matrix that starts at zero,

        d = softplus(dt + dt_bias),   S <- exp(-exp(A_log) d) S + d B x^T,   y = S^T C + D x

    The joined heads are multiplied by silu(z), divided by their root mean square in ``norm_groups`` equal runs, multiplied
    by a gain, and W_o adds the result into the residual row.

    A request keeps in its slot the last taps - 1 rows that the convolution read and, behind them, S, all float32.  A prompt
    portion runs its tokens in order from the stored state and leaves the new one there, a decode step is a portion of one
    token.  The projection and the convolved rows are of the compute type; everything behind them is float32 (csrc/ssd.cu).

    With one norm group a step of few rows leaves the gated rows in float32 and the output product norms them in its own
    prologue.

    params: hidden_size, n_heads, v_dim, state, groups, norm_groups, taps, eps, init_std, out_init_std; tensors in, conv,
    conv.b, dt_bias, A_log, D, norm, o.
    """

    graph_safe = True
    accepts_deferred_norm = True
    takes_result_factor = True

    MAX_STATE = 512

    def __init__(self, params, prefix, env):
        super().__init__(params, prefix, env)
        p = self.params
        if p["n_heads"] % p["groups"]:
            raise ValueError("state_space: groups must divide the heads")
        if not (0 < p["state"] <= self.MAX_STATE) or not (0 < p["v_dim"] <= 1024):
            raise ValueError("state_space: at most 512 x 1024 numbers of state per head")
        if not (isinstance(p["taps"], int) and 1 <= p["taps"] <= 16):
            raise ValueError("state_space: a convolution has 1 to 16 taps")
        self.inner = p["n_heads"] * p["v_dim"]
        if not (0 < p["norm_groups"] <= 64) or self.inner % p["norm_groups"]:
            raise ValueError("state_space: between 1 and 64 norm groups that divide the joined heads")
        self.channels = self.inner + 2 * p["groups"] * p["state"]
        self.kept = (p["taps"] - 1) * self.channels
        self.rows = self.inner + self.channels + p["n_heads"]

    def state_need(self):
        p = self.params
        return StateNeed((padded(self.kept) + p["n_heads"] * p["state"] * p["v_dim"],), "float32")

    def param_specs(self):
        p, std = self.params, self.params.get("init_std", 0.02)
        H = p["n_heads"]
        return [(ParamSpec(self._n("in"), (self.rows, p["hidden_size"]), "matmul"), ("normal", std)),
                (ParamSpec(self._n("conv"), (self.channels, p["taps"]), "vector"), ("normal", p["taps"] ** -0.5)),
                (ParamSpec(self._n("conv.b"), (self.channels,), "vector"), ("normal", 0.1)),
                (ParamSpec(self._n("dt_bias"), (H,), "vector"), ("normal", 1.0)),
                (ParamSpec(self._n("A_log"), (H,), "vector"), ("normal", 1.0)),
                (ParamSpec(self._n("D"), (H,), "vector"), ("ones_plus_normal", 0.1)),
                (ParamSpec(self._n("norm"), (self.inner,), "vector"), ("ones_plus_normal", 0.1)),
                (ParamSpec(self._n("o"), (p["hidden_size"], self.inner), "matmul"), ("normal", p.get("out_init_std", std)))]

    def bind(self, tensors):
        t = lambda name: tensors[self._n(name)].contiguous()
        w_in = t("in")
        # a row of the product ends on a multiple of eight numbers: rows of zeros behind dt's
        self.w_in = torch.cat([w_in, w_in.new_zeros((-self.rows % 8, w_in.shape[1]))], dim=0).contiguous()
        self.conv, self.conv_bias = t("conv"), t("conv.b")
        self.dt_bias, self.a_log, self.d, self.gain, self.w_o = t("dt_bias"), t("A_log"), t("D"), t("norm"), t("o")
        # the norm in front of the output product, in the form that a product can take into its prologue
        self.norm = LayerNorm(dict(width=self.inner, eps=self.params["eps"], name="norm", has_mean=False, has_bias=False), "",
                              self.env)
        self.norm.weight, self.norm.bias = self.gain, None

    def forward(self, x, residual, ctx, layer):
        p, ops, dtype, device = self.params, self.env.ops, self.env.dtype, residual.device
        tokens, H, P, G, N = x.shape[0], p["n_heads"], p["v_dim"], p["groups"], p["state"]
        raw = ops.empty((tokens, self.w_in.shape[0]), dtype, device)
        ops.linear(x, self.w_in, None, raw)
        conv = ops.empty((tokens, self.channels), dtype, device)
        ops.short_conv(raw[:, self.inner:self.inner + self.channels], self.conv, p["taps"], self.channels,
                       layer.state[:, :self.kept] if self.kept else None, ctx, conv, bias=self.conv_bias, act="silu")
        at = padded(self.kept)
        own = state_share(layer, at, layer.state.shape[1] - at)
        few = tokens <= ops.FUSED_NORM_ROWS and p["norm_groups"] == 1
        gated = ops.empty((tokens, self.inner), torch.float32 if few else dtype, device)
        ops.ssd(conv, raw, (0, self.inner, self.inner + G * N, 0, self.inner + self.channels), self.a_log, self.dt_bias, self.d,
                own.state, ctx, gated, H, G, N, P)
        if few:
            normed = DeferredNorm(self.norm, gated)
        else:
            normed = ops.empty((tokens, self.inner), dtype, device)
            ops.group_rms_norm(gated, self.gain, float(p["eps"]), p["norm_groups"], normed)
        ops.linear(normed, self.w_o, None, residual, accumulate=True, factor=self.result_factor)
