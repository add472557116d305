"""The Miberax architecture through the engine's host logic on the CPU (plain PyTorch kernels),
against the plain float64 model: configuration, checkpoint layout, the parts of a layer, every way
of cutting requests into steps, long decoding and greedy generation through the scheduler."""

import copy

import pytest
import torch

import plain_miberax as pm
import traces
from conftest import MIBERAX_TINY
from plain_ops import PlainOps

NAMES = sorted(MIBERAX_TINY)


def cpu_runner(folder, name, num_pages, max_num_seqs=4, max_len=512):
    from llmserve_b200.engine.runner import ModelRunner, load_model

    _, _, model = load_model(folder, "float32", "cpu", PlainOps(), max_len)
    return ModelRunner(model, page_tokens=MIBERAX_TINY[name]["page_tokens"], num_pages=num_pages,
                       max_model_len=max_len, max_num_seqs=max_num_seqs)


def test_config_round_trip_and_refusals():
    from llmserve_b200.config import ConfigError, architecture_for
    from llmserve_b200.config.miberax import MiberaxConfig

    for name in NAMES:
        d = MIBERAX_TINY[name]["config"]
        assert architecture_for(d).name == "Miberax"
        cfg = MiberaxConfig.from_dict(d)
        assert cfg.to_dict() == d and MiberaxConfig.from_dict(cfg.to_dict()) == cfg
    d = MIBERAX_TINY["M1"]["config"]
    cfg = MiberaxConfig.from_dict(d)
    assert cfg.norm_groups == 4 and cfg.layers[2].mlp is None and cfg.layers[0].left.rot_factor == 2.0
    assert cfg.layers[1].mlp.keep == 2 and cfg.layers[1].mlp.identity == 1 and cfg.layers[1].right.conv == 2
    # what may be absent: the mask, the rotation, the groups, identity experts, the scale, the shared expert
    b = copy.deepcopy(d)
    m = b["layers"][1]
    for k in ("groups", "identity", "scale"):
        m["mlp"]["router"].pop(k)
    m["mlp"].pop("shared")
    m["mixer"]["left"].pop("mask")
    m["mixer"]["left"].pop("rot")
    l = MiberaxConfig.from_dict(b).layers[1]
    assert (l.mlp.groups, l.mlp.keep, l.mlp.identity, l.mlp.scale, l.mlp.shared_ff) == (1, 1, 0, 1.0, 0)
    assert l.left.chunk == 0 and l.left.rot_dims == 0

    def broken(change):
        b = copy.deepcopy(d)
        change(b)
        with pytest.raises(ConfigError):
            MiberaxConfig.from_dict(b)

    broken(lambda b: b["layers"][0].update(type="retention"))
    broken(lambda b: b["layers"][0]["mixer"].pop("right"))
    broken(lambda b: b["layers"][0]["mixer"]["left"].pop("scale"))
    broken(lambda b: b["layers"][0]["mixer"]["left"].update(window=3))
    broken(lambda b: b["layers"][0]["mixer"]["left"].update(kv_heads=3))
    broken(lambda b: b["layers"][0]["mixer"]["left"]["rot"].update(dims=26))
    broken(lambda b: b["layers"][0]["mixer"]["left"]["rot"].update(scaling={"kind": "other"}))
    broken(lambda b: b["layers"][0]["mixer"]["right"].update(conv=0))
    broken(lambda b: b["layers"][0]["mixer"]["right"].update(kv_heads=3))
    broken(lambda b: b["layers"][1]["mlp"]["router"]["groups"].update(count=4))
    broken(lambda b: b["layers"][1]["mlp"]["router"]["groups"].update(keep=4))
    broken(lambda b: b["layers"][1]["mlp"]["router"].update(top=5))  # more than the kept groups hold
    broken(lambda b: b["layers"][1]["mlp"]["expert"].pop("limit"))
    broken(lambda b: b["layers"][0]["mlp"].update(kind="gated"))
    broken(lambda b: b["norm"].update(groups=7))
    broken(lambda b: b.pop("norm"))


def test_plan_is_prenorm_blocks_of_two_mixers_side_by_side():
    from llmserve_b200.config.miberax import MiberaxConfig
    from llmserve_b200.models.miberax import miberax_plan

    plan = miberax_plan(MiberaxConfig.from_dict(MIBERAX_TINY["M1"]["config"]))
    assert [l.kind for l in plan.layers] == ["prenorm"] * 3 and plan.tie_head
    l = plan.layers[0]
    assert l.mixer.kind == "parallel" and [b.kind for b in l.mixer.branches] == ["attention", "gated_delta_rule"]
    assert l.mixer.coefficients == (0.5, 0.5) and l.norm_in.groups == 4 and plan.final_norm.groups == 4
    assert l.mixer.branches[0].position.pairing == "neighbours" and l.mixer.branches[0].chunk == 21
    assert l.feed_forward.activation == "poly_norm" and plan.layers[2].feed_forward is None
    e = plan.layers[1].feed_forward
    assert e.router_weights == "softmax_of_all" and e.identity_experts == 1 and e.shared_limit == 1.3 and e.groups == 3


def test_branches_share_one_product_and_a_chunk_bounds_the_pages(miberax_dirs):
    runner = cpu_runner(miberax_dirs["M1"], "M1", 16)
    mixer = runner.model.blocks[0].mixer
    assert mixer.shared_weight is not None and all(c % 8 == 0 for c in mixer.columns)
    for b, c in zip(mixer.branches, mixer.columns):  # views, not copies
        assert b.input_weight.data_ptr() == mixer.shared_weight[c].data_ptr()
    assert sorted(g.window for g in runner.manager.groups) == [16, 21, 40]


def test_checkpoint_errors_are_reported_together(miberax_dirs, tmp_path):
    from safetensors.torch import load_file, save_file

    from llmserve_b200.engine.runner import load_model
    from llmserve_b200.weights.loader import CheckpointError

    t = load_file(str(miberax_dirs["M1"] / "model.safetensors"))
    t.pop("l0.mix.right.A_log")
    t["l2.mlp.up"] = torch.zeros(8, 96)  # the layer has no feed-forward
    t["l1.mlp.correction"] = torch.zeros(5)  # the identity expert has one too
    save_file(t, str(tmp_path / "model.safetensors"))
    (tmp_path / "config.json").write_text((miberax_dirs["M1"] / "config.json").read_text())
    with pytest.raises(CheckpointError) as e:
        load_model(tmp_path, "float32", "cpu", PlainOps(), 64)
    assert e.value.missing == ["l0.mix.right.A_log"] and e.value.unexpected == ["l2.mlp.up"]
    assert [w[0] for w in e.value.wrong_shape] == ["l1.mlp.correction"]


def test_neighbouring_pairs_are_halves_after_a_reordering():
    from llmserve_b200.parts.positions import neighbours_to_halves

    order = neighbours_to_halves(10, 6)
    assert order == [0, 2, 4, 1, 3, 5, 6, 7, 8, 9] and sorted(order) == list(range(10))
    x = torch.randn(5, 1, 10, dtype=torch.float64)
    ref = pm.rotate_neighbours(x, torch.arange(5), 6, 100.0, 2.0)[..., order]
    y = x[..., order]
    a = torch.arange(5, dtype=torch.float64)[:, None] * (100.0 ** (-2.0 * torch.arange(3, dtype=torch.float64) / 6) / 2.0)
    c, s = a.cos()[:, None], a.sin()[:, None]
    got = torch.cat([y[..., :3] * c - y[..., 3:6] * s, y[..., 3:6] * c + y[..., :3] * s, y[..., 6:]], -1)
    assert torch.allclose(got, ref)


def test_options_that_go_together_are_checked():
    from llmserve_b200.parts.base import BuildEnv
    from llmserve_b200.parts.delta_rule import GatedDeltaRule, GatedDeltaRuleSpec
    from llmserve_b200.parts.moe import RoutedExperts, RoutedExpertsSpec
    from llmserve_b200.parts.norms import RMSNorm, RMSNormSpec

    env = BuildEnv(ops=PlainOps(), dtype=torch.float32, device=torch.device("cpu"), max_positions=8)
    with pytest.raises(ValueError):
        RMSNorm(RMSNormSpec(10, 1e-5, groups=3), env)
    with pytest.raises(ValueError):
        GatedDeltaRule(GatedDeltaRuleSpec(16, 3, 2, 4, 4, 2, 1e-5), env)
    ok = dict(hidden_size=16, num_experts=6, top=2, expert_size=8, weight_on="output", router_weights="softmax_of_all")
    RoutedExperts(RoutedExpertsSpec(**ok, groups=2, keep_groups=1, identity_experts=2), env)
    for bad in (dict(groups=4), dict(groups=3, keep_groups=4), dict(groups=6, keep_groups=1)):
        with pytest.raises(ValueError):
            RoutedExperts(RoutedExpertsSpec(**ok, **bad), env)
    with pytest.raises(ValueError):
        RoutedExperts(RoutedExpertsSpec(16, 6, 2, 8, identity_experts=1), env)


LENGTHS = {"M1": [5, 70, 1, 33, 49, 126, 2], "M2": [2, 40, 9, 64, 17, 90], "M3": [3, 80, 18, 110]}


@pytest.fixture(scope="module")
def expected(miberax_dirs):
    out = {}
    for name in NAMES:
        reqs = traces.make_requests(LENGTHS[name], MIBERAX_TINY[name]["config"]["vocab"], seed=5)
        out[name] = (reqs, {r: pm.model_logits(miberax_dirs[name], t) for r, t in reqs.items()})
    return out


@pytest.mark.parametrize("name,mode", [("M1", "whole"), ("M1", "portions"), ("M1", "mixed"), ("M2", "decode_tail"),
                                       ("M2", "mixed"), ("M3", "portions")])
def test_every_way_of_cutting_matches_plain(miberax_dirs, expected, name, mode):
    reqs, exp = expected[name]
    runner = cpu_runner(miberax_dirs[name], name, traces.tokens_needed(reqs) // MIBERAX_TINY[name]["page_tokens"])
    got = traces.replay(runner, getattr(traces, mode)(reqs))
    traces.compare(got, exp, atol=2e-4, rtol=2e-5)
    assert runner.manager.usage() == 0.0


def test_long_decoding_from_the_first_token_on_few_pages(miberax_dirs):
    """110 tokens one by one from position 0: chunks begin and end among decoded tokens and give their
    pages back, the states are carried through every step."""
    reqs = traces.make_requests([110], 131, seed=21)
    exp = {r: pm.model_logits(miberax_dirs["M2"], t) for r, t in reqs.items()}
    runner = cpu_runner(miberax_dirs["M2"], "M2", 6)  # 48 of 110 tokens fit
    traces.compare(traces.replay(runner, traces.decode_tail(reqs, tail=110)), exp, atol=2e-4, rtol=2e-5)


def test_greedy_generation_through_the_scheduler(miberax_dirs):
    from llmserve_b200 import LLM, SamplingParams

    prompts = [[5, 9, 100, 31, 7], list(range(40, 57)), [3] * 33, [100, 2]]
    m = LLM(str(miberax_dirs["M1"]), dtype="float32", device="cpu", ops=PlainOps(), block_size=16, num_kv_blocks=24,
            max_model_len=128, max_num_seqs=3, max_num_batched_tokens=24)
    outs = m.generate(prompts, SamplingParams(temperature=0.0, max_tokens=6, ignore_eos=True))
    for o, p in zip(outs, prompts):
        assert o.outputs[0].token_ids == pm.greedy(miberax_dirs["M1"], p, 6), p


@pytest.mark.parametrize("name", ["M1", "M3"])
def test_steps_that_want_some_rows_or_none(miberax_dirs, name):
    wanted_subsets(lambda: cpu_runner(miberax_dirs[name], name, 16), miberax_dirs[name], MIBERAX_TINY[name]["config"]["vocab"])


def wanted_subsets(make_runner, folder, vocab, atol=2e-4, rtol=2e-5):
    """Steps that want some rows, one row or none: the model's last norm then reads only those rows, and
    the branches a last layer without feed-forward leaves are summed without it."""
    from llmserve_b200.engine.batch import StepEntry

    reqs = traces.make_requests([41, 30], vocab, seed=13)
    exp = {r: pm.model_logits(folder, t) for r, t in reqs.items()}
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
