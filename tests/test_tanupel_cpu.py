"""The Tanupel architecture through the engine's host logic on the CPU (plain PyTorch kernels),
against the plain float64 model: configuration, checkpoint layout, the run order of a loop, the parts of a
layer, every way of cutting requests into steps, long decoding and greedy generation through the scheduler."""

import copy
import json
import math

import pytest
import torch

import plain_tanupel as pt
import traces
from conftest import TANUPEL_TINY
from plain_ops import PlainOps

NAMES = sorted(TANUPEL_TINY)


def cpu_runner(folder, name, num_pages, max_num_seqs=4, max_len=512):
    from llmserve_b200.engine.runner import ModelRunner, load_model

    _, _, model = load_model(folder, "float32", "cpu", PlainOps(), max_len)
    return ModelRunner(model, page_tokens=TANUPEL_TINY[name]["page_tokens"], num_pages=num_pages,
                       max_model_len=max_len, max_num_seqs=max_num_seqs)


def test_config_round_trip_and_refusals():
    from llmserve_b200.config import ConfigError, architecture_for
    from llmserve_b200.config.tanupel import TanupelConfig

    for name in NAMES:
        d = TANUPEL_TINY[name]["config"]
        assert architecture_for(d).name == "Tanupel"
        cfg = TanupelConfig.from_dict(d)
        assert cfg.to_dict() == d and TanupelConfig.from_dict(cfg.to_dict()) == cfg
    d = TANUPEL_TINY["T1"]["config"]
    cfg = TanupelConfig.from_dict(d)
    assert cfg.loop == (1, 3, 2) and cfg.layers[2].mlp is None and cfg.layers[1].mixer.left.rot.scaling == "linear"
    assert cfg.layers[0].mixer.rot.scaling == "llama3" and cfg.layers[0].mixer.softcap == 4.0
    # what may be absent or null: the loop, a rotation, its scaling, a soft cap, the ranks
    b = copy.deepcopy(d)
    b["loop"] = None
    b["layers"][0]["mixer"].update(rot=None, softcap=None)
    b["layers"][1]["mixer"]["left"]["rot"]["scaling"] = None
    b["layers"][1]["mixer"]["right"].pop("decay_rank")
    cfg = TanupelConfig.from_dict(b)
    assert cfg.loop is None and cfg.layers[0].mixer.rot is None and cfg.layers[0].mixer.softcap == 0.0
    assert cfg.layers[1].mixer.left.rot.scaling == "default" and cfg.layers[1].mixer.right.decay_rank == 0
    from llmserve_b200.models.tanupel import tanupel_plan

    with pytest.raises(ValueError, match="inner sizes"):
        tanupel_plan(cfg)

    def broken(change):
        b = copy.deepcopy(d)
        change(b)
        with pytest.raises(ConfigError):
            TanupelConfig.from_dict(b)

    broken(lambda b: b["layers"][0].update(type="retention"))
    broken(lambda b: b["layers"][1]["mixer"].pop("right_scale"))
    broken(lambda b: b["layers"][0]["mixer"].pop("scale"))
    broken(lambda b: b["layers"][0]["mixer"].update(mask={"size": 3}))
    broken(lambda b: b["layers"][0]["mixer"].update(kv_heads=3))
    broken(lambda b: b["layers"][0]["mixer"].update(softcap=-1.0))
    broken(lambda b: b["layers"][0]["mixer"]["rot"].update(dims=26))
    broken(lambda b: b["layers"][0]["mixer"]["rot"]["scaling"].pop("low"))
    broken(lambda b: b["layers"][0]["mixer"]["rot"]["scaling"].update(kind="other"))
    broken(lambda b: b["layers"][1]["mixer"]["right"].update(conv=0))
    broken(lambda b: b["layers"][1]["mixer"]["right"].update(kv_heads=3))
    broken(lambda b: b["layers"][1]["mlp"]["router"].update(top=6))
    broken(lambda b: b["layers"][1]["mlp"].update(shared={"ff": 4}))
    broken(lambda b: b["layers"][0]["mlp"].update(kind="gated"))
    broken(lambda b: b["loop"].update(stop=1))
    broken(lambda b: b["loop"].update(stop=5))
    broken(lambda b: b["loop"].update(times=0))
    broken(lambda b: b.pop("residual_mult"))


def test_plan_is_shared_norm_blocks_in_a_run_order_with_a_loop():
    from llmserve_b200.config.tanupel import TanupelConfig
    from llmserve_b200.models.tanupel import tanupel_plan

    plan = tanupel_plan(TanupelConfig.from_dict(TANUPEL_TINY["T1"]["config"]))
    assert [l.kind for l in plan.layers] == ["shared_norm"] * 4 and not plan.tie_head and plan.embed_scale == 3.5
    assert [(e.layer, e.cache, e.vector) for e in plan.run_order] == [
        (0, 0, None), (1, 1, 0), (2, 2, None), (1, 3, 1), (2, 4, None), (3, 5, None)]
    assert plan.run_vectors == 2 and plan.layers[0].coefficient == 0.7 and plan.final_norm.unit_offset
    l = plan.layers[1]
    assert l.mixer.kind == "parallel" and [b.kind for b in l.mixer.branches] == ["attention", "gated_delta_rule"]
    assert l.mixer.coefficients == (0.8, 1.4) and not l.mixer.normed and l.mixer.branches[0].softcap == 6.0
    d = l.mixer.branches[1]
    assert (d.decay_rank, d.gate_rank, d.gate_activation) == (8, 24, "sigmoid")
    assert not l.feed_forward.normalise_weights and l.feed_forward.correction and plan.layers[2].feed_forward is None
    no_loop = tanupel_plan(TanupelConfig.from_dict(TANUPEL_TINY["T3"]["config"]))
    assert [(e.layer, e.vector) for e in no_loop.run_order] == [(0, None), (1, None), (2, None)] and no_loop.run_vectors == 0


def test_plan_checks_its_vectors():
    import dataclasses

    from llmserve_b200.config.tanupel import TanupelConfig
    from llmserve_b200.models.plan import RunEntry
    from llmserve_b200.models.tanupel import tanupel_plan

    plan = tanupel_plan(TanupelConfig.from_dict(TANUPEL_TINY["T1"]["config"]))
    with pytest.raises(ValueError):
        dataclasses.replace(plan, run_order=(RunEntry(0, 0, 2),)).validate()
    with pytest.raises(ValueError):
        dataclasses.replace(plan, residual_streams=2).validate()


def test_every_pass_has_its_own_cache_and_branches_share_one_product(tanupel_dirs):
    runner = cpu_runner(tanupel_dirs["T1"], "T1", 16)
    assert len(runner.model.cache_needs()) == 6
    mixer = runner.model.blocks[1].mixer
    assert mixer.shared_weight is not None and all(c % 8 == 0 for c in mixer.columns)
    for b, c in zip(mixer.branches, mixer.columns):  # views, not copies
        assert b.input_weight.data_ptr() == mixer.shared_weight[c].data_ptr()
    right = mixer.branches[1]
    assert right.inner == 24 and right.inner_col % 8 == 0 and tuple(right.inner_weight.shape) == (2, 128, 24)


def test_ranks_come_from_the_tensors_shapes(tanupel_dirs, tmp_path):
    from llmserve_b200.config.tanupel import TanupelConfig

    d = json.loads((tanupel_dirs["T2"] / "config.json").read_text())
    for l in d["layers"]:
        if l["type"] == "parallel":
            del l["mixer"]["right"]["decay_rank"], l["mixer"]["right"]["gate_rank"]
    (tmp_path / "config.json").write_text(json.dumps(d))
    (tmp_path / "model.safetensors").write_bytes((tanupel_dirs["T2"] / "model.safetensors").read_bytes())
    cfg = TanupelConfig.from_pretrained(tmp_path)
    assert cfg.to_dict() == TANUPEL_TINY["T2"]["config"]


def test_checkpoint_errors_are_reported_together(tanupel_dirs, tmp_path):
    from safetensors.torch import load_file, save_file

    from llmserve_b200.engine.runner import load_model
    from llmserve_b200.weights.loader import CheckpointError

    t = load_file(str(tanupel_dirs["T1"] / "model.safetensors"))
    t.pop("l1.mix.right.A_log")
    t.pop("loop.step")
    t["l2.mlp.up"] = torch.zeros(8, 96)  # the layer has no feed-forward
    t["l1.mix.right.dt_bias"] = torch.zeros(4)  # one per head and key channel is needed
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text((tanupel_dirs["T1"] / "config.json").read_text())
    with pytest.raises(CheckpointError) as e:
        load_model(tmp_path, "float32", "cpu", PlainOps(), 64)
    assert e.value.missing == ["l1.mix.right.A_log", "loop.step"] and e.value.unexpected == ["l2.mlp.up"]
    assert [w[0] for w in e.value.wrong_shape] == ["l1.mix.right.dt_bias"]


def test_scaled_frequencies_leave_short_waves_divide_long_ones_and_blend_between():
    from llmserve_b200.parts.positions import RotarySpec, rotary_inverse_frequencies

    rot = {"base": 1000.0, "dims": 20, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 200}}
    f = pt.frequencies(rot)
    plain = pt.frequencies({"base": 1000.0, "dims": 20})
    waves = 2 * math.pi / plain
    assert (f[waves < 50] == plain[waves < 50]).all() and (waves < 50).any()
    assert torch.allclose(f[waves > 200], plain[waves > 200] / 8) and (waves > 200).any()
    mid = (waves >= 50) & (waves <= 200)
    assert mid.any() and ((f[mid] < plain[mid]) & (f[mid] > plain[mid] / 8)).all()
    got = rotary_inverse_frequencies(RotarySpec(head_dim=20, theta=1000.0, scaling_type="llama3", factor=8.0,
                                                low_freq_factor=1.0, high_freq_factor=4.0, original_max_positions=200))
    assert torch.allclose(got, f, rtol=1e-12)
    linear = rotary_inverse_frequencies(RotarySpec(head_dim=20, theta=1000.0, scaling_type="linear", factor=8.0))
    assert torch.allclose(linear, pt.frequencies(dict(rot, scaling={"factor": 8.0})), rtol=1e-12)


def test_options_that_go_together_are_checked():
    from llmserve_b200.parts.base import BuildEnv
    from llmserve_b200.parts.delta_rule import GatedDeltaRule, GatedDeltaRuleSpec
    from llmserve_b200.parts.moe import RoutedExperts, RoutedExpertsSpec

    env = BuildEnv(ops=PlainOps(), dtype=torch.float32, device=torch.device("cpu"), max_positions=8)
    for bad in (dict(decay_rank=4), dict(gate_rank=4), dict(gate_activation="relu")):
        with pytest.raises(ValueError):
            GatedDeltaRule(GatedDeltaRuleSpec(16, 2, 2, 4, 4, 2, 1e-5, **bad), env)
    with pytest.raises(ValueError):
        RoutedExperts(RoutedExpertsSpec(16, 6, 2, 8, normalise_weights=False), env)


def test_pending_adds_and_a_vector_before_a_run():
    """A vector joins what is already pending, whatever that is, and everything is added exactly once."""
    from llmserve_b200.parts.base import PendingAdds, with_row

    ops, x0, y = PlainOps(), torch.randn(3, 8), torch.randn(3, 8)
    row = torch.randn(8)
    x = x0.clone()
    p = with_row(ops, x, None, row)
    assert p.resolve() is None and torch.allclose(x, x0 + row)
    p.resolve()
    assert torch.allclose(x, x0 + row)
    x = x0.clone()
    with_row(ops, x, y, row).resolve()
    assert torch.allclose(x, x0 + y + row)
    x = x0.clone()
    p = with_row(ops, x, PendingAdds(ops, x, [(0.5, y), (-2.0, y)]), row)
    with_row(ops, x, p, row).resolve()  # a second vector: the first is added before
    assert torch.allclose(x, x0 - 1.5 * y + 2 * row, atol=1e-6)


def test_any_mixer_and_feed_forward_fit_the_shared_norm_block():
    """Parts that know nothing of coefficients go through the default ``forward_into``."""
    from llmserve_b200.parts.attention import AttentionSpec
    from llmserve_b200.parts.base import BuildEnv, FeedForward, Mixer, PendingAdds
    from llmserve_b200.parts.blocks import SharedNormBlock, SharedNormBlockSpec
    from llmserve_b200.parts.norms import RMSNormSpec
    from llmserve_b200.parts.positions import NoPositionSpec

    ops = PlainOps()
    env = BuildEnv(ops=ops, dtype=torch.float32, device=torch.device("cpu"), max_positions=8)

    class Half(Mixer):
        def forward(self, h, step, cache):
            return 0.5 * h

    class Twice(FeedForward):
        def forward(self, h, step):
            return 2 * h

    mixer = AttentionSpec(hidden_size=8, num_heads=1, num_kv_heads=1, head_dim=16, scale=1.0, position=NoPositionSpec())
    block = SharedNormBlock(SharedNormBlockSpec(norm=RMSNormSpec(8, 1e-5), mixer=mixer, coefficient=0.25), env)
    block.norm.weight = torch.ones(8)
    block.mixer, block.feed_forward = Half(None, env), Twice(None, env)
    x = torch.randn(3, 8)
    h = pt.unit_rms(x.double(), 1e-5)
    ref = x.double() + 0.25 * 2.5 * h
    x1, pending = block.forward(x.clone(), None, None, None)
    assert isinstance(pending, PendingAdds) and pending.resolve() is None
    assert torch.allclose(x1.double(), ref, atol=1e-5)


LENGTHS = {"T1": [5, 70, 1, 33, 49, 90, 2], "T2": [2, 40, 9, 64, 17, 80], "T3": [3, 80, 18, 110]}


@pytest.fixture(scope="module")
def expected(tanupel_dirs):
    out = {}
    for name in NAMES:
        reqs = traces.make_requests(LENGTHS[name], TANUPEL_TINY[name]["config"]["vocab"], seed=5)
        out[name] = (reqs, {r: pt.model_logits(tanupel_dirs[name], t) for r, t in reqs.items()})
    return out


@pytest.mark.parametrize("name,mode", [("T1", "whole"), ("T1", "portions"), ("T1", "mixed"), ("T2", "decode_tail"),
                                       ("T2", "mixed"), ("T3", "portions")])
def test_every_way_of_cutting_matches_plain(tanupel_dirs, expected, name, mode):
    reqs, exp = expected[name]
    runner = cpu_runner(tanupel_dirs[name], name, traces.tokens_needed(reqs) // TANUPEL_TINY[name]["page_tokens"])
    got = traces.replay(runner, getattr(traces, mode)(reqs))
    traces.compare(got, exp, atol=2e-4, rtol=2e-5)
    assert runner.manager.usage() == 0.0


def test_mechanisms_that_must_show_in_the_logits(tanupel_dirs):
    """Each mechanism left out of the plain model changes its logits by far more than any tolerance used here."""
    cfg, w = pt.load(tanupel_dirs["T1"])
    tokens = traces.make_requests([60], 167, seed=9)["r0"]
    ref = pt.forward(tokens, w, cfg)

    def change(edit):
        c, v = copy.deepcopy(cfg), dict(w)
        edit(c, v)
        return (pt.forward(tokens, v, c) - ref).abs().max().item() / ref.abs().max().item()

    edits = {
        "the vectors of the passes": lambda c, v: v.update({"loop.step": v["loop.step"] * 0}),
        "one pass fewer": lambda c, v: c["loop"].update(times=1),
        "a soft cap": lambda c, v: c["layers"][0]["mixer"].pop("softcap"),
        "a soft cap beside the delta rule": lambda c, v: c["layers"][1]["mixer"]["left"].pop("softcap"),
        "the scaling of frequencies": lambda c, v: c["layers"][0]["mixer"]["rot"].pop("scaling"),
        "a factor of the pair": lambda c, v: c["layers"][1]["mixer"].update(right_scale=1.0),
        "the constant on what a layer adds": lambda c, v: c.update(residual_mult=1.0),
        "a query norm's weight": lambda c, v: v.update({"l2.mix.q.norm": v["l2.mix.q.norm"] * 0 + 1.6}),
        "decays that differ by channel": lambda c, v: v.update(
            {"l1.mix.right.dt_bias": v["l1.mix.right.dt_bias"] * 0 + v["l1.mix.right.dt_bias"].mean()}),
        "the convolution": lambda c, v: v.update({"l1.mix.right.v.conv": v["l1.mix.right.v.conv"].flip(1)}),
        "the correction's absence from the weights": lambda c, v: v.update({"l1.mlp.correction": v["l1.mlp.correction"] + 0.5 * torch.eye(5, dtype=torch.float64)[0]}),
    }
    for what, edit in edits.items():
        assert change(edit) > 5e-3, what


def test_long_decoding_from_the_first_token(tanupel_dirs):
    reqs = traces.make_requests([110], 131, seed=21)
    exp = {r: pt.model_logits(tanupel_dirs["T2"], t) for r, t in reqs.items()}
    runner = cpu_runner(tanupel_dirs["T2"], "T2", 14)
    traces.compare(traces.replay(runner, traces.decode_tail(reqs, tail=110)), exp, atol=2e-4, rtol=2e-5)


@pytest.mark.parametrize("name", NAMES)
def test_steps_that_want_some_rows_or_none(tanupel_dirs, name):
    wanted_subsets(lambda: cpu_runner(tanupel_dirs[name], name, 16), tanupel_dirs[name], TANUPEL_TINY[name]["config"]["vocab"])


def wanted_subsets(make_runner, folder, vocab, atol=2e-4, rtol=2e-5):
    """Steps that want some rows, one row or none: the model's last norm then reads only those rows, and what the
    last layer left is added without it."""
    from llmserve_b200.engine.batch import StepEntry

    reqs = traces.make_requests([41, 30], vocab, seed=13)
    exp = {r: pt.model_logits(folder, t) for r, t in reqs.items()}
    runner = make_runner()
    a, b = reqs["r0"], reqs["r1"]
    steps = [[("r0", a[:17], [3, 16]), ("r1", b[:9], [])],
             [("r0", a[17:18], []), ("r1", b[9:22], [])],
             [("r0", a[18:19], [0]), ("r1", b[22:23], [])],
             [("r0", a[19:41], [21]), ("r1", b[23:30], [6, 2])]]
    at = {"r0": 0, "r1": 0}
    for entries in steps:
        logits = runner.run([StepEntry(r, t, w) for r, t, w in entries]).float().cpu()
        row = 0
        for r, t, w in entries:
            for k in w:
                ref = exp[r][at[r] + k]
                assert (logits[row] - ref).abs().max().item() <= atol + rtol * ref.abs().max().item(), (r, at[r] + k)
                row += 1
            at[r] += len(t)
        assert row == logits.shape[0]


def test_greedy_generation_through_the_scheduler(tanupel_dirs):
    from llmserve_b200 import LLM, SamplingParams

    prompts = [[5, 9, 100, 31, 7], list(range(40, 57)), [3] * 33, [100, 2]]
    m = LLM(str(tanupel_dirs["T1"]), dtype="float32", device="cpu", ops=PlainOps(), block_size=16, num_kv_blocks=24,
            max_model_len=128, max_num_seqs=3, max_num_batched_tokens=24)
    outs = m.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    for o, p in zip(outs, prompts):
        assert o.outputs[0].token_ids == pt.greedy(tanupel_dirs["T1"], p, 6), p
