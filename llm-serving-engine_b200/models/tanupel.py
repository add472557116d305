"""The Tanupel architecture as data: which parts each layer has and where its tensors come from.

Every layer is a ``shared_norm`` block: its mixer and its feed-forward read the same normed rows (a
weight stored around zero), and a constant times their sum is added to the residual stream. The
mixer is one of

* ``attention``: grouped query heads; queries and keys normed over the whole projection, part of each
  head rotated (optionally with scaled frequencies), optionally a soft cap on the scores;
* ``parallel``: such an attention beside the gated delta rule with a decay per key channel and a
  sigmoid gate, both made through small matrices; their outputs are summed with a constant each.

The feed-forward is gated and dense; or routed experts (softmax over all scores, a correction for the
choice, the scores themselves as weights); or absent.

The embedded tokens are multiplied by a constant. A run of layers may be repeated with the same
weights: every pass has a cache of its own, and a learned vector per pass is added to the residual
stream before the pass begins. The output projection is a matrix of its own.

Checkpoint tensors are named ``l<i>.<part>``; the matrices of one product are concatenated along
their rows (q | k | v; q | k | v | b | a1 | g1; gate | up; all experts' gate | up; all experts' down).
"""

from __future__ import annotations

from ..config.tanupel import CorrectedExpertsConfig, TanupelConfig
from ..parts.attention import AttentionSpec
from ..parts.blocks import SharedNormBlockSpec
from ..parts.delta_rule import GatedDeltaRuleSpec
from ..parts.feed_forward import SwiGLUSpec
from ..parts.moe import RoutedExpertsSpec
from ..parts.norms import RMSNormSpec
from ..parts.parallel import ParallelMixerSpec
from ..parts.positions import NoPositionSpec, RotarySpec
from .plan import CheckpointLayout, ModelPlan, ParamSource, RunEntry, Source


def _attention(m, w: int, eps: float) -> AttentionSpec:
    position = NoPositionSpec()
    if m.rot is not None and m.rot.dims:
        r = m.rot
        position = RotarySpec(head_dim=r.dims, theta=r.base, scaling_type=r.scaling, factor=r.factor,
                              low_freq_factor=r.low, high_freq_factor=r.high, original_max_positions=r.original)
    return AttentionSpec(hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, head_dim=m.dim, value_dim=m.vdim,
                         scale=m.scale, position=position, qk_norm_eps=eps, qk_norm_scope="row", softcap=m.softcap)


def _delta_rule(m, w: int, eps: float) -> GatedDeltaRuleSpec:
    if min(m.decay_rank, m.gate_rank) < 1:
        raise ValueError("parallel: the inner sizes of the decay and gate matrices are not known (they are read from "
                         "the checkpoint's tensor shapes, or given as decay_rank and gate_rank)")
    return GatedDeltaRuleSpec(hidden_size=w, num_heads=m.heads, num_kv_heads=m.kv_heads, key_dim=m.dim,
                              value_dim=m.vdim, conv=m.conv, eps=eps, query_scale=m.dim ** -0.5,
                              decay_rank=m.decay_rank, gate_rank=m.gate_rank, gate_activation="sigmoid")


def _mixer(l, w: int, eps: float):
    if l.type == "attention":
        return _attention(l.mixer, w, eps)
    m = l.mixer
    return ParallelMixerSpec(hidden_size=w, names=("left", "right"), normed=False,
                             branches=(_attention(m.left, w, eps), _delta_rule(m.right, w, eps)),
                             coefficients=(m.left_scale, m.right_scale))


def _feed_forward(m, w: int):
    if m is None:
        return None
    if isinstance(m, CorrectedExpertsConfig):
        return RoutedExpertsSpec(w, m.experts, m.top, m.ff, router_weights="softmax_of_all", weight_on="output",
                                 correction=True, normalise_weights=False)
    return SwiGLUSpec(w, m.ff)


def tanupel_run_order(cfg: TanupelConfig) -> tuple[RunEntry, ...]:
    """Every run has a cache layer of its own; the first layer of pass t of the loop adds vector t."""
    n = len(cfg.layers)
    start, stop, times = cfg.loop or (n, n, 0)
    runs = [(i, None) for i in range(start)]
    runs += [(i, t if i == start else None) for t in range(times) for i in range(start, stop)]
    runs += [(i, None) for i in range(stop, n)]
    return tuple(RunEntry(i, k, vector) for k, (i, vector) in enumerate(runs))


def tanupel_plan(cfg: TanupelConfig) -> ModelPlan:
    w, eps = cfg.hidden_size, cfg.norm_eps
    norm = RMSNormSpec(w, eps, unit_offset=True)
    layers = tuple(SharedNormBlockSpec(norm=norm, mixer=_mixer(l, w, eps), feed_forward=_feed_forward(l.mlp, w),
                                       coefficient=cfg.residual_mult) for l in cfg.layers)
    return ModelPlan(vocab_size=cfg.vocab_size, hidden_size=w, layers=layers, run_order=tanupel_run_order(cfg),
                     final_norm=norm, tie_head=False, embed_scale=cfg.embed_scale,
                     run_vectors=cfg.loop[2] if cfg.loop else 0)


def _attention_entries(m, src: str, dst: str, w: int) -> list[ParamSource]:
    q, k, v = m.heads * m.dim, m.kv_heads * m.dim, m.kv_heads * m.vdim
    return [
        ParamSource(dst + "qkv.weight", (Source(src + "q", (q, w)), Source(src + "k", (k, w)), Source(src + "v", (v, w)))),
        ParamSource(dst + "q_norm.weight", (Source(src + "q.norm", (q,)),), "scale"),
        ParamSource(dst + "k_norm.weight", (Source(src + "k.norm", (k,)),), "scale"),
        ParamSource(dst + "o.weight", (Source(src + "o", (w, m.heads * m.vdim)),)),
    ]


def _delta_entries(m, src: str, dst: str, w: int) -> list[ParamSource]:
    qk, v = m.kv_heads * m.dim, m.heads * m.vdim
    return [
        ParamSource(dst + "in.weight", (Source(src + "q", (qk, w)), Source(src + "k", (qk, w)), Source(src + "v", (v, w)),
                                        Source(src + "b", (m.heads, w)), Source(src + "a1", (m.decay_rank, w)),
                                        Source(src + "g1", (m.gate_rank, w)))),
        ParamSource(dst + "conv.weight", (Source(src + "q.conv", (qk, m.conv)), Source(src + "k.conv", (qk, m.conv)),
                                          Source(src + "v.conv", (v, m.conv))), "scale"),
        ParamSource(dst + "A_log", (Source(src + "A_log", (m.heads,)),), "offset"),
        ParamSource(dst + "dt_bias", (Source(src + "dt_bias", (m.heads * m.dim,)),), "offset"),
        ParamSource(dst + "decay_out.weight", (Source(src + "a2", (m.heads * m.dim, m.decay_rank)),)),
        ParamSource(dst + "gate_out.weight", (Source(src + "g2", (v, m.gate_rank)),)),
        ParamSource(dst + "norm.weight", (Source(src + "norm", (m.vdim,)),), "scale"),
        ParamSource(dst + "o.weight", (Source(src + "o", (w, v)),)),
    ]


def tanupel_checkpoint_layout(cfg: TanupelConfig) -> CheckpointLayout:
    w = cfg.hidden_size
    entries = [
        ParamSource("embed.weight", (Source("embed", (cfg.vocab_size, w)),), "embedding"),
        ParamSource("final_norm.weight", (Source("final.norm", (w,)),), "offset"),
        ParamSource("head.weight", (Source("head", (cfg.vocab_size, w)),)),
    ]
    if cfg.loop:
        entries.append(ParamSource("run_vectors", (Source("loop.step", (cfg.loop[2], w)),), "offset"))
    for i, l in enumerate(cfg.layers):
        src, dst, m = f"l{i}.", f"layers.{i}.", l.mixer
        entries.append(ParamSource(dst + "norm.weight", (Source(src + "norm1", (w,)),), "offset"))
        if l.type == "attention":
            entries += _attention_entries(m, src + "mix.", dst + "mixer.", w)
        else:
            entries += _attention_entries(m.left, src + "mix.left.", dst + "mixer.left.", w)
            entries += _delta_entries(m.right, src + "mix.right.", dst + "mixer.right.", w)
        if l.mlp is None:
            continue
        m, fs, fd = l.mlp, src + "mlp.", dst + "feed_forward."
        if isinstance(m, CorrectedExpertsConfig):
            entries += [
                ParamSource(fd + "router.weight", (Source(fs + "router", (m.experts, w)),), "matrix32"),
                ParamSource(fd + "router.correction", (Source(fs + "correction", (m.experts,)),), "offset"),
                ParamSource(fd + "experts.gate_up.weight", tuple(
                    Source(f"{fs}e{e}.{part}", (m.ff, w)) for e in range(m.experts) for part in ("gate", "up"))),
                ParamSource(fd + "experts.down.weight", tuple(Source(f"{fs}e{e}.down", (w, m.ff)) for e in range(m.experts))),
            ]
        else:
            entries += [
                ParamSource(fd + "gate_up.weight", (Source(fs + "gate", (m.ff, w)), Source(fs + "up", (m.ff, w)))),
                ParamSource(fd + "down.weight", (Source(fs + "down", (w, m.ff)),)),
            ]
    return CheckpointLayout(entries=tuple(entries))
