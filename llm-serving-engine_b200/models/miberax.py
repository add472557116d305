"""The Miberax architecture as data: which parts each layer has and where its tensors come from.

Every layer is a ``prenorm`` block whose norms work on equal parts of the row one by one. Its mixer
is ``parallel``: two mixers that read the same input, each output normed over the width, half of
each summed:

* ``left``: grouped query heads with rotary positions on neighbouring dims (part of each head, all
  frequencies divided by a constant), every query limited to the keys of its own chunk of positions;
* ``right``: the gated delta rule with a short convolution, a norm per head and a SiLU gate.

The feed-forward is ``Wdown act(Wup h)`` with a polynomial of norms as ``act``; or routed experts (softmax
over all scores, a correction for the choice, groups of experts, identity experts, clamped gated
experts with the weight on the output, a shared expert behind a sigmoid gate); or absent. The
output projection is the embedding table.

Checkpoint tensors are named ``l<i>.<part>``; the matrices of one product are concatenated along
their rows (q | k | v; q | k | v | g | b | a; all experts' gate | up; all experts' down; router | sg).
"""

from __future__ import annotations

from ..config.miberax import GroupedExpertsConfig, MiberaxConfig
from ..parts.attention import AttentionSpec
from ..parts.blocks import PreNormBlockSpec
from ..parts.delta_rule import GatedDeltaRuleSpec
from ..parts.feed_forward import MLPSpec
from ..parts.moe import RoutedExpertsSpec
from ..parts.norms import RMSNormSpec
from ..parts.parallel import ParallelMixerSpec
from ..parts.positions import NoPositionSpec, RotarySpec
from .plan import CheckpointLayout, ModelPlan, ParamSource, RunEntry, Source


def _left(m, w: int) -> AttentionSpec:
    position = NoPositionSpec()
    if m.rot_dims:
        position = RotarySpec(head_dim=m.rot_dims, theta=m.rot_base, scaling_type="linear", factor=m.rot_factor,
                              pairing="neighbours")
    return AttentionSpec(hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                         scale=m.scale, position=position, chunk=m.chunk)


def _right(m, w: int, eps: float) -> GatedDeltaRuleSpec:
    return GatedDeltaRuleSpec(hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim,
                              value_dim=m.vdim, conv=m.conv, eps=eps, query_scale=m.dim ** -0.5)


def _feed_forward(m, w: int, eps: float):
    if m is None:
        return None
    if isinstance(m, GroupedExpertsConfig):
        return RoutedExpertsSpec(
            w, m.experts, m.top, m.ff, m.shared_ff, activation="clamped_glu", router_weights="softmax_of_all",
            weight_on="output", correction=True, groups=m.groups, keep_groups=m.keep, router_scale=m.scale,
            identity_experts=m.identity, limit=m.limit, shared_limit=m.shared_limit)
    return MLPSpec(w, m.ff, activation="poly_norm", eps=eps)


def miberax_plan(cfg: MiberaxConfig) -> ModelPlan:
    w, eps = cfg.hidden_size, cfg.norm_eps
    norm = RMSNormSpec(w, eps, groups=cfg.norm_groups)
    layers = []
    for l in cfg.layers:
        mixer = ParallelMixerSpec(hidden_size=w, names=("left", "right"), branches=(_left(l.left, w), _right(l.right, w, eps)),
                                  coefficients=(0.5, 0.5), eps=eps)
        ff = _feed_forward(l.mlp, w, eps)
        layers.append(PreNormBlockSpec(norm_in=norm, mixer=mixer, norm_post=norm if ff is not None else None,
                                       feed_forward=ff))
    return ModelPlan(vocab_size=cfg.vocab_size, hidden_size=w, layers=tuple(layers),
                     run_order=tuple(RunEntry(i, i) for i in range(len(layers))), final_norm=norm, tie_head=True)


def miberax_checkpoint_layout(cfg: MiberaxConfig) -> CheckpointLayout:
    w = cfg.hidden_size
    entries = [
        ParamSource("embed.weight", (Source("embed", (cfg.vocab_size, w)),), "embedding"),
        ParamSource("final_norm.weight", (Source("final.norm", (w,)),), "scale"),
    ]
    ignored = []
    for i, l in enumerate(cfg.layers):
        src, dst = f"l{i}.", f"layers.{i}."
        entries.append(ParamSource(dst + "norm_in.weight", (Source(src + "norm1", (w,)),), "scale"))
        m, ms, md = l.left, src + "mix.left.", dst + "mixer.left."
        entries += [
            ParamSource(md + "qkv.weight", (Source(ms + "q", (m.heads * m.dim, w)), Source(ms + "k", (m.kv_heads * m.dim, w)),
                                            Source(ms + "v", (m.kv_heads * m.vdim, w)))),
            ParamSource(md + "o.weight", (Source(ms + "o", (w, m.heads * m.vdim)),)),
            ParamSource(dst + "mixer.out.left.weight", (Source(ms + "out", (w,)),), "scale"),
        ]
        m, ms, md = l.right, src + "mix.right.", dst + "mixer.right."
        qk, vg = m.kv_heads * m.dim, m.heads * m.vdim
        entries += [
            ParamSource(md + "in.weight", (Source(ms + "q", (qk, w)), Source(ms + "k", (qk, w)), Source(ms + "v", (vg, w)),
                                           Source(ms + "g", (vg, w)), Source(ms + "b", (m.heads, w)),
                                           Source(ms + "a", (m.heads, w)))),
            ParamSource(md + "conv.weight", (Source(ms + "q.conv", (qk, m.conv)), Source(ms + "k.conv", (qk, m.conv)),
                                             Source(ms + "v.conv", (vg, m.conv))), "scale"),
            ParamSource(md + "A_log", (Source(ms + "A_log", (m.heads,)),), "offset"),
            ParamSource(md + "dt_bias", (Source(ms + "dt_bias", (m.heads,)),), "offset"),
            ParamSource(md + "norm.weight", (Source(ms + "norm", (m.vdim,)),), "scale"),
            ParamSource(md + "o.weight", (Source(ms + "o", (w, vg)),)),
            ParamSource(dst + "mixer.out.right.weight", (Source(ms + "out", (w,)),), "scale"),
        ]
        if l.mlp is None:
            ignored.append(src + "norm2")  # a file may carry the unused norm of a layer without feed-forward
            continue
        entries.append(ParamSource(dst + "norm_post.weight", (Source(src + "norm2", (w,)),), "scale"))
        m, fs, fd = l.mlp, src + "mlp.", dst + "feed_forward."
        if not isinstance(m, GroupedExpertsConfig):
            entries += [
                ParamSource(fd + "up.weight", (Source(fs + "up", (m.ff, w)),)),
                ParamSource(fd + "coefficients", (Source(fs + "act", (4,)),), "scale"),
                ParamSource(fd + "down.weight", (Source(fs + "down", (w, m.ff)),)),
            ]
            continue
        choices = m.experts + m.identity
        router = [Source(fs + "router", (choices, w))]
        if m.shared_ff:
            router.append(Source(fs + "shared.sg", (1, w)))
            entries += [
                ParamSource(fd + "shared.gate_up.weight", (Source(fs + "shared.gate", (m.shared_ff, w)),
                                                           Source(fs + "shared.up", (m.shared_ff, w)))),
                ParamSource(fd + "shared.down.weight", (Source(fs + "shared.down", (w, m.shared_ff)),)),
            ]
        entries += [
            ParamSource(fd + "router.weight", tuple(router), "matrix32"),
            ParamSource(fd + "router.correction", (Source(fs + "correction", (choices,)),), "offset"),
            ParamSource(fd + "experts.gate_up.weight", tuple(
                Source(f"{fs}e{e}.{part}", (m.ff, w)) for e in range(m.experts) for part in ("gate", "up"))),
            ParamSource(fd + "experts.down.weight", tuple(Source(f"{fs}e{e}.down", (w, m.ff)) for e in range(m.experts))),
        ]
    return CheckpointLayout(entries=tuple(entries), ignored_names=tuple(ignored))
