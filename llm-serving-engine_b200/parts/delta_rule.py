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
  values that all heads share; the concatenated heads are multiplied by ``silu(Wg h)`` (or its
  sigmoid) and projected by ``Wo``.

``decay_rank`` and ``gate_rank`` (both or neither): decays per channel. ``g = exp(-exp(A_log) softplus(A2 (A1 h) +
dt_bias))`` is then one number per value head *and key channel* (row d of S is multiplied by ``g_d``),
made from the token through two small matrices of inner size ``decay_rank``, and the gate is made
the same way, ``G2 (G1 h)`` with inner size ``gate_rank``.

One matrix product makes q | k | v | gate | b | a, or q | k | v | b | A1 h | G1 h; both second products
of the ranks are one launch. Convolution, norms, decay, step size, the
recurrence and the gate run in float32 inside the kernels, whatever the compute dtype of the
products is. Kept per request: ``S^T`` as ``[heads, value_dim, key_dim]`` and the last ``conv - 1``
inputs of the convolution, ``[conv - 1, channels]`` (nothing for a convolution of one tap).
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from .attention import rows_to_whole_vectors
from .base import MIXERS, Mixer, ParamDecl, StateNeed, add_projected, project_into


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
    decay_rank: int = 0  # > 0: decays per key channel through two matrices of this inner size
    gate_rank: int = 0  # > 0 (together with decay_rank): the gate likewise
    gate_activation: str = "silu"  # or "sigmoid"
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
        if (spec.decay_rank > 0) != (spec.gate_rank > 0) or min(spec.decay_rank, spec.gate_rank) < 0:
            raise ValueError("gated delta rule: decay_rank and gate_rank are both positive or both zero")
        if spec.gate_activation not in ("silu", "sigmoid"):
            raise ValueError("gated delta rule: unknown activation of the gate")
        self.qk = spec.num_kv_heads * spec.key_dim
        self.vg = spec.num_heads * spec.value_dim
        self.channels = 2 * self.qk + self.vg
        self.by_channel = spec.decay_rank > 0
        # by_channel: the columns of A1 h and G1 h in the product, each filled up to `inner` whole vectors
        self.inner = -(-max(spec.decay_rank, spec.gate_rank) // 8) * 8
        self.inner_col = -(-(self.channels + spec.num_heads) // 8) * 8

    def param_decls(self):
        s = self.spec
        rows = (s.num_heads + s.decay_rank + s.gate_rank) if self.by_channel else (self.vg + 2 * s.num_heads)
        decls = {
            # rows: q, k, v, gate, b, a; or q, k, v, b, A1, G1
            "in.weight": ParamDecl((self.channels + rows, s.hidden_size), "matrix"),
            "conv.weight": ParamDecl((self.channels, s.conv), "scale"),
            "A_log": ParamDecl((s.num_heads,), "offset"),
            "dt_bias": ParamDecl((s.num_heads * (s.key_dim if self.by_channel else 1),), "offset"),
            "norm.weight": ParamDecl((s.value_dim,), "scale"),
            "o.weight": ParamDecl((s.hidden_size, self.vg), "matrix"),
        }
        if self.by_channel:
            decls["decay_out.weight"] = ParamDecl((s.num_heads * s.key_dim, s.decay_rank), "matrix")
            decls["gate_out.weight"] = ParamDecl((self.vg, s.gate_rank), "matrix")
        return decls

    def bind(self, params):
        s = self.spec
        w = params["in.weight"]
        if self.by_channel:
            head = self.channels + s.num_heads
            full = w.new_zeros(self.inner_col + 2 * self.inner, w.shape[1])
            full[:head] = w[:head]
            full[self.inner_col : self.inner_col + s.decay_rank] = w[head : head + s.decay_rank]
            at = self.inner_col + self.inner
            full[at : at + s.gate_rank] = w[head + s.decay_rank :]
            w = full
            # both second matrices as a product per half: [2, larger of both row counts, inner]
            rows = max(s.num_heads * s.key_dim, self.vg)
            self.inner_weight = w.new_zeros(2, rows, self.inner)
            self.inner_weight[0, : s.num_heads * s.key_dim, : s.decay_rank] = params["decay_out.weight"]
            self.inner_weight[1, : self.vg, : s.gate_rank] = params["gate_out.weight"]
        self.input_weight = rows_to_whole_vectors(w)
        self.conv_taps = params["conv.weight"].t().contiguous()  # [taps, channels]: a tap's channels side by side
        self.A_log = params["A_log"]
        self.dt_bias = params["dt_bias"]
        self.norm_weight = params["norm.weight"].repeat(s.num_heads).contiguous()  # the same for every head
        self.o_weight = params["o.weight"]

    def cache_need(self):
        s = self.spec
        state = StateNeed((s.num_heads, s.value_dim, s.key_dim), torch.float32)
        return (state, StateNeed((s.conv - 1, self.channels), torch.float32)) if s.conv > 1 else (state,)

    accepts_deferral = True

    def forward(self, h, step, cache, may_defer=False):
        proj = self.ops.linear(h, self.input_weight, None, out_dtype=torch.float32)
        return self.forward_projected(proj, 0, step, cache, may_defer)

    def forward_into(self, h, step, cache, x, coefficient):
        proj = self.ops.linear(h, self.input_weight, None, out_dtype=torch.float32)
        return self.forward_projected(proj, 0, step, cache, add_to=(x, coefficient))

    def forward_projected(self, proj, col0, step, cache, may_defer=False, add_to=None):
        """As ``forward`` from the float32 product with the input, whose columns for this mixer start at ``col0``;
        with ``add_to = (x, coefficient)`` as ``forward_into``."""
        s, ops = self.spec, self.ops
        sizes = dict(num_heads=s.num_heads, num_kv_heads=s.num_kv_heads, key_dim=s.key_dim, value_dim=s.value_dim)
        conv = dict(conv=self.conv_taps, conv_state=cache.states[1] if s.conv > 1 else None)
        if self.by_channel:
            zg = ops.inner_linear(proj, col0 + self.inner_col, self.inner_weight, self.env.dtype)
            qkv, scal, decay = ops.delta_inputs(
                proj, col0, **conv, A_log=self.A_log, dt_bias=self.dt_bias, query_scale=s.query_scale, step=step,
                decay_logits=zg, **sizes)
            o = ops.delta_rule(qkv, scal, state=cache.states[0], step=step, decay=decay, **sizes)
            gate, gate_col = zg, self.inner_weight.shape[1]
        else:
            qkv, scal = ops.delta_inputs(
                proj, col0, **conv, A_log=self.A_log, dt_bias=self.dt_bias, query_scale=s.query_scale, step=step, **sizes)
            o = ops.delta_rule(qkv, scal, state=cache.states[0], step=step, **sizes)
            gate, gate_col = proj, col0 + self.channels
        y = ops.gated_group_norm(
            o, gate, gate_offset=gate_col, group=s.value_dim, weight=self.norm_weight, eps=s.eps,
            gate_activation=s.gate_activation, out_dtype=self.env.dtype)
        if add_to is not None:
            return add_projected(ops, y, self.o_weight, None, *add_to)
        return project_into(ops, y, self.o_weight, None, self.env.residual_dtype, None, may_defer)
