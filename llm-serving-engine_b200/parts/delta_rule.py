"""The gated delta rule: linear attention that corrects its state instead of only adding to it.

Per value head, with a state ``S [key_dim, value_dim]``, a decay ``g`` and a step size ``beta`` per token:

    S <- g S;   u = beta (v - S^T k);   S <- S + k u^T;   o = S^T q

so that a key which was written before has its old value taken out before the new one goes in.
Around it:

* q, k and v pass a short causal convolution over time per channel (``conv`` taps, zeros before the
  start of the sequence) and silu; q and k are made unit vectors per head (``x / sqrt(sum x^2 +
  1e-6)``), q is multiplied by ``query_scale``; a value head reads key head ``h // (heads / kv_heads)``;
* ``beta = sigmoid(Wb h)``, ``g = exp(-exp(A_log) softplus(Wa h + dt_bias))``, one number per value head;
* each head's ``o`` is divided by its root mean square and multiplied by a weight of ``value_dim``
  values that all heads share; the concatenated heads are multiplied by ``silu(Wg h)`` and projected
  by ``Wo``.

One matrix product makes q | k | v | gate | b | a. Convolution, norms, decay, step size, the
recurrence and the gate run in float32 inside the kernels, whatever the compute dtype of the
products is. Kept per request: ``S^T`` as ``[heads, value_dim, key_dim]`` and the last ``conv - 1``
inputs of the convolution, ``[conv - 1, channels]`` (nothing for a convolution of one tap).
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .attention import rows_to_whole_vectors
from .base import MIXERS, Mixer, ParamDecl, StateNeed, project_into


@dataclass(frozen=True)
class GatedDeltaRuleSpec:
    hidden_size: int
    num_heads: int
    num_kv_heads: int
    key_dim: int
    value_dim: int
    conv: int  # taps of the short convolution, the current token's included
    eps: float
    query_scale: float = 1.0
    kind: str = "gated_delta_rule"


@MIXERS.register("gated_delta_rule")
class GatedDeltaRule(Mixer):
    keeps_running_state = True

    def __init__(self, spec: GatedDeltaRuleSpec, env) -> None:
        super().__init__(spec, env)
        if spec.num_heads % spec.num_kv_heads:
            raise ValueError("gated delta rule: heads must be a multiple of kv_heads")
        if spec.conv < 1:
            raise ValueError("gated delta rule: the convolution has at least one tap")
        self.qk = spec.num_kv_heads * spec.key_dim
        self.vg = spec.num_heads * spec.value_dim
        self.channels = 2 * self.qk + self.vg

    def param_decls(self):
        s = self.spec
        return {
            # rows: q, k, v, gate, b, a
            "in.weight": ParamDecl((self.channels + self.vg + 2 * s.num_heads, s.hidden_size), "matrix"),
            "conv.weight": ParamDecl((self.channels, s.conv), "scale"),
            "A_log": ParamDecl((s.num_heads,), "offset"),
            "dt_bias": ParamDecl((s.num_heads,), "offset"),
            "norm.weight": ParamDecl((s.value_dim,), "scale"),
            "o.weight": ParamDecl((s.hidden_size, self.vg), "matrix"),
        }

    def bind(self, params):
        self.input_weight = rows_to_whole_vectors(params["in.weight"])
        self.conv_taps = params["conv.weight"].t().contiguous()  # [taps, channels]: a tap's channels side by side
        self.A_log = params["A_log"]
        self.dt_bias = params["dt_bias"]
        self.norm_weight = params["norm.weight"].repeat(self.spec.num_heads).contiguous()  # the same for every head
        self.o_weight = params["o.weight"]

    def cache_need(self):
        s = self.spec
        state = StateNeed((s.num_heads, s.value_dim, s.key_dim), torch.float32)
        return (state, StateNeed((s.conv - 1, self.channels), torch.float32)) if s.conv > 1 else (state,)

    accepts_deferral = True

    def forward(self, h, step, cache, may_defer=False):
        proj = self.ops.linear(h, self.input_weight, None, out_dtype=torch.float32)
        return self.forward_projected(proj, 0, step, cache, may_defer)

    def forward_projected(self, proj, col0, step, cache, may_defer=False):
        """As ``forward`` from the float32 product with the input, whose columns for this mixer start at ``col0``."""
        s, ops = self.spec, self.ops
        sizes = dict(num_heads=s.num_heads, num_kv_heads=s.num_kv_heads, key_dim=s.key_dim, value_dim=s.value_dim)
        qkv, scal = ops.delta_inputs(
            proj, col0, conv=self.conv_taps, conv_state=cache.states[1] if s.conv > 1 else None, A_log=self.A_log,
            dt_bias=self.dt_bias, query_scale=s.query_scale, step=step, **sizes)
        o = ops.delta_rule(qkv, scal, state=cache.states[0], step=step, **sizes)
        y = ops.gated_group_norm(
            o, proj, gate_offset=col0 + self.channels, group=s.value_dim, weight=self.norm_weight, eps=s.eps,
            gate_activation="silu", out_dtype=self.env.dtype)
        return project_into(ops, y, self.o_weight, None, self.env.residual_dtype, None, may_defer)
