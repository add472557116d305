"""Mixers side by side: every branch reads the same input; their outputs are normed one by one
and summed with fixed coefficients.

    out = sum_b coefficient_b * w_b * a_b / sqrt(mean(a_b^2) + eps),      a_b = branch_b(h)

``normed=False``: the branches' outputs are summed as they are, ``sum_b coefficient_b * a_b``.

Branches that can start from a product made for them (``input_weight``, ``forward_projected``) share
one: their matrices are laid one below the other when the weights are bound.

Each branch is a mixer of its own kind with its own cache need; the cache layer of the block holds
all of them (pages for one, states for others), and each branch sees its own part of it.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any

import torch

from .base import MIXERS, BranchMix, Mixer, ParamDecl, PendingAdds, count_states, flatten_needs, has_pages


@dataclass(frozen=True)
class ParallelMixerSpec:
    hidden_size: int
    names: tuple[str, ...]
    branches: tuple[Any, ...]  # mixer specs
    coefficients: tuple[float, ...]
    eps: float = 0.0
    normed: bool = True
    kind: str = "parallel"


@MIXERS.register("parallel")
class ParallelMixer(Mixer):
    def __init__(self, spec: ParallelMixerSpec, env) -> None:
        super().__init__(spec, env)
        if not (len(spec.names) == len(spec.branches) == len(spec.coefficients)) or not spec.branches:
            raise ValueError("names, branches and coefficients must have one entry per branch")
        self.children = {n: MIXERS.build(b, env) for n, b in zip(spec.names, spec.branches)}
        self.branches = list(self.children.values())
        # which part of the shared cache layer each branch sees
        self._parts = []
        first = 0
        for b in self.branches:
            need = b.cache_need()
            self._parts.append((has_pages(need), first, count_states(need)))
            first += count_states(need)

    def param_decls(self):
        out = {}
        for name, child in self.children.items():
            for pname, decl in child.param_decls().items():
                out[f"{name}.{pname}"] = decl
            if self.spec.normed:
                out[f"out.{name}.weight"] = ParamDecl((self.spec.hidden_size,), "scale")
        return out

    def bind(self, params):
        self.out_weights = []
        for name, child in self.children.items():
            prefix = name + "."
            child.bind({k[len(prefix):]: v for k, v in params.items() if k.startswith(prefix)})
            if self.spec.normed:
                self.out_weights.append(params[f"out.{name}.weight"])
        self._share_product()

    def _share_product(self):
        """One product with the input for all branches, if every branch can take its columns of it.
        Every branch starts on a column that is a multiple of 8; what the branches hold of their
        own becomes a view of the shared matrix."""
        self.shared_weight = None
        weights = [getattr(b, "input_weight", None) for b in self.branches]
        if len(weights) < 2 or any(w is None for w in weights):
            return
        padded, self.columns, at = [], [], 0
        for w in weights:
            self.columns.append(at)
            extra = (-w.shape[0]) % 8
            padded += [w] + ([w.new_zeros(extra, w.shape[1])] if extra else [])
            at += w.shape[0] + extra
        self.input_weight = torch.cat(padded, 0).contiguous()

    @property
    def input_weight(self):
        """The matrix of the branches' one product with the input (None: they make their own)."""
        return self.shared_weight

    @input_weight.setter
    def input_weight(self, w):
        self.shared_weight = w
        for b, c in zip(self.branches, self.columns):
            b.input_weight = w[c : c + b.input_weight.shape[0]]

    def cache_need(self):
        return tuple(n for b in self.branches for n in flatten_needs(b.cache_need()))

    accepts_deferral = True

    def forward_into(self, h, step, cache, x, coefficient):
        if self.spec.normed:
            return [(coefficient, self.forward(h, step, cache).resolve())]
        if self.shared_weight is not None:
            proj = self.ops.linear(h, self.shared_weight, None, out_dtype=torch.float32)
            return self.forward_projected(proj, 0, step, cache, add_to=(x, coefficient))
        items = []
        for b, c, part in zip(self.branches, self.spec.coefficients, self._parts):
            items += b.forward_into(h, step, cache.part(*part), x, coefficient * c)
        return items

    def forward_projected(self, proj, col0, step, cache, add_to):
        """``forward_into`` (``add_to = (x, coefficient)``) from the float32 product with the input, whose columns for
        this mixer start at ``col0``."""
        x, coefficient = add_to
        items = []
        for b, c, at, part in zip(self.branches, self.spec.coefficients, self.columns, self._parts):
            items += b.forward_projected(proj, col0 + at, step, cache.part(*part), add_to=(x, coefficient * c))
        return items

    def forward(self, h, step, cache, may_defer=False):
        if not self.spec.normed:
            x = torch.zeros(h.shape[0], self.spec.hidden_size, dtype=torch.float32, device=h.device)
            PendingAdds(self.ops, x, self.forward_into(h, step, cache, x, 1.0)).resolve()
            return x
        outs = []
        if self.shared_weight is not None:
            proj = self.ops.linear(h, self.shared_weight, None, out_dtype=torch.float32)
            for b, c, (pages, first, n) in zip(self.branches, self.columns, self._parts):
                outs.append(b.forward_projected(proj, c, step, cache.part(pages, first, n), may_defer=may_defer))
            return BranchMix(self.ops, outs, self.out_weights, tuple(self.spec.coefficients), self.spec.eps)
        for b, (pages, first, n) in zip(self.branches, self._parts):
            defer = may_defer and getattr(b, "accepts_deferral", False)
            a = (b.forward(h, step, cache.part(pages, first, n), may_defer=True) if defer
                 else b.forward(h, step, cache.part(pages, first, n)))
            # a branch's product that is not converted yet stays so only if the caller takes such
            outs.append(a.resolve() if hasattr(a, "resolve") and not defer else a)
        return BranchMix(self.ops, outs, self.out_weights, tuple(self.spec.coefficients), self.spec.eps)
