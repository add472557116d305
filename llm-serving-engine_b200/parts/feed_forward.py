"""Dense gated feed-forward (src/llmserve/models/transformer.py:62-71).

    gu = h @ Wgu^T          rows of Wgu: gate (first I rows), then up (last I rows)
    y  = (act(gate) * up) @ Wdown^T,     act = silu: g / (1 + exp(-g)), or
                                         gelu_tanh: 0.5 g (1 + tanh(sqrt(2/pi) (g + 0.044715 g^3)))

No biases. The activation is computed in float32 (src/llmserve/kernels/csrc/fused_ops.cpp:75-91).

``activation="clamped_glu"`` combines the two halves otherwise: ``g sigmoid(1.702 g) (u + 1)`` with ``g =
min(gate, limit)`` and ``u = clamp(up, -limit, limit)``.

``mlp`` is the ungated form, ``y = Wdown act(Wup h)``, with ``act`` one of ``relu2`` (the square of
relu), ``relu``, ``gelu_tanh``, ``silu``, or ``poly_norm``: with four learned numbers a, b, c, e,
``a N(z) + b N(z^2) + c N(z^3) + e``, powers taken element by element and ``N`` a token's whole vector
divided by its root mean square (``eps`` of the spec), in float32.
"""

from __future__ import annotations

from dataclasses import dataclass

from .base import FEED_FORWARDS, FeedForward, ParamDecl, add_projected, project_into


GATED_ACTIVATIONS = ("silu", "gelu_tanh", "clamped_glu")


@dataclass(frozen=True)
class SwiGLUSpec:
    hidden_size: int
    intermediate_size: int
    kind: str = "swiglu"
    activation: str = "silu"  # or "gelu_tanh", "clamped_glu"
    limit: float = 0.0  # of clamped_glu


@FEED_FORWARDS.register("swiglu")
class SwiGLU(FeedForward):
    def param_decls(self):
        s = self.spec
        return {
            "gate_up.weight": ParamDecl((2 * s.intermediate_size, s.hidden_size), "matrix"),
            "down.weight": ParamDecl((s.hidden_size, s.intermediate_size), "matrix"),
        }

    def __init__(self, spec: SwiGLUSpec, env) -> None:
        super().__init__(spec, env)
        if spec.activation not in GATED_ACTIVATIONS:
            raise ValueError(f"gated feed-forward: activation {spec.activation!r} is not known")
        self._options = {} if spec.activation != "clamped_glu" else {"limit": spec.limit}

    def bind(self, params):
        self.gate_up_weight = params["gate_up.weight"]
        self.down_weight = params["down.weight"]

    accepts_residual = True

    def forward_into(self, h, step, x, coefficient):
        return add_projected(self.ops, self._inner(h), self.down_weight, None, x, coefficient)

    @property
    def input_weight(self):
        """The matrix of this part's product with its input, where a block may make it part of a larger one."""
        return self.gate_up_weight

    @input_weight.setter
    def input_weight(self, w):
        self.gate_up_weight = w

    def forward_projected(self, proj, col0, add_to):
        """``forward_into`` (``add_to = (x, coefficient)``) from the float32 product with the input, whose columns for
        this part start at ``col0``."""
        a = self.ops.silu_mul(proj, out_dtype=self.env.dtype, activation=self.spec.activation,
                              columns=(col0, 2 * self.spec.intermediate_size), **self._options)
        return add_projected(self.ops, a, self.down_weight, None, *add_to)

    def _inner(self, h):
        if self.spec.activation == "silu":
            return self.ops.gated_silu(h, self.gate_up_weight, None, out_dtype=self.env.dtype)
        return self.ops.gated_silu(h, self.gate_up_weight, None, out_dtype=self.env.dtype,
                                   activation=self.spec.activation, **self._options)

    def forward(self, h, step, residual=None, may_defer=False):
        return project_into(self.ops, self._inner(h), self.down_weight, None, self.env.residual_dtype, residual, may_defer)


PLAIN_ACTIVATIONS = ("relu2", "relu", "gelu_tanh", "silu")


@dataclass(frozen=True)
class MLPSpec:
    hidden_size: int
    intermediate_size: int
    activation: str = "relu2"  # or another of PLAIN_ACTIVATIONS, or "poly_norm"
    eps: float = 0.0  # of poly_norm
    kind: str = "mlp"


@FEED_FORWARDS.register("mlp")
class MLP(FeedForward):
    accepts_residual = True

    def __init__(self, spec: MLPSpec, env) -> None:
        super().__init__(spec, env)
        if spec.activation not in PLAIN_ACTIVATIONS + ("poly_norm",):
            raise ValueError(f"feed-forward: activation {spec.activation!r} is not known")

    def param_decls(self):
        s = self.spec
        decls = {
            "up.weight": ParamDecl((s.intermediate_size, s.hidden_size), "matrix"),
            "down.weight": ParamDecl((s.hidden_size, s.intermediate_size), "matrix"),
        }
        if s.activation == "poly_norm":
            decls["coefficients"] = ParamDecl((4,), "scale")
        return decls

    def bind(self, params):
        self.up_weight = params["up.weight"]
        self.down_weight = params["down.weight"]
        self.coefficients = params.get("coefficients")

    def forward_into(self, h, step, x, coefficient):
        return add_projected(self.ops, self._inner(h), self.down_weight, None, x, coefficient)

    def _inner(self, h):
        if self.spec.activation == "poly_norm":
            return self.ops.poly_norm_linear(h, self.up_weight, self.coefficients, self.spec.eps, self.env.dtype)
        return self.ops.activated_linear(h, self.up_weight, self.spec.activation, self.env.dtype)

    def forward(self, h, step, residual=None, may_defer=False):
        return project_into(self.ops, self._inner(h), self.down_weight, None, self.env.residual_dtype, residual, may_defer)
