"""The Miberax parts on the GPU: each kernel against the plain float64 function of its mechanism,
then the model through the step function and through generation, against the plain model."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_miberax as pm
import traces
from conftest import MIBERAX_TINY
from test_miberax_cpu import wanted_subsets

pytestmark = pytest.mark.gpu

F = torch.float64
NAMES = sorted(MIBERAX_TINY)
BOTH = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def ops():
    from llmserve_b200.ops import get_ops

    return get_ops("cuda")


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def i32(a):
    return torch.tensor(np.asarray(a), dtype=torch.int32).cuda()


def batch(q_lens, starts, slots):
    """The step arrays of a ragged batch (sequence i: q_lens[i] rows from position starts[i])."""
    cu = np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int32)
    host = SimpleNamespace(q_lens=np.asarray(q_lens, dtype=np.int32),
                           ctx_lens=(np.asarray(starts) + np.asarray(q_lens)).astype(np.int32))
    return SimpleNamespace(
        cu_q=i32(cu), ctx_lens=i32(host.ctx_lens), state_slots=i32(slots),
        token_seq=i32(np.repeat(np.arange(len(q_lens)), q_lens)),
        positions=i32(np.concatenate([np.arange(s, s + n) for s, n in zip(starts, q_lens)])),
        host=host, decode_splits=0,
        max_decode_ctx=int(max([s + n for s, n in zip(starts, q_lens) if n == 1], default=0)))


def close(got, ref, tol, what=""):
    err = (got.double().cpu() - ref.double()).abs().max().item()
    bound = tol * max(1.0, ref.abs().max().item())
    assert err <= bound, f"{what}: {err:.3e} > {bound:.3e}"


# ----------------------------------------------------------------------------- norms
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W,groups", [(5, 96, 4), (3, 70, 1), (4, 70, 7), (7, 2048, 2), (2, 120, 60), (1, 66, 2)])
def test_parts_of_a_row_are_normed_one_by_one(ops, dtype, T, W, groups):
    x, r, w = rnd(T, W, seed=1), rnd(T, W, seed=2), 1 + rnd(W, seed=3, scale=0.3)
    x[:, : W // groups] *= 30  # one part much larger than the others: a norm of the whole row would show
    tol = 3e-6 if dtype == torch.float32 else 6e-3
    eps = 0.01
    xd = x.cuda()
    got = ops.add_rmsnorm(xd, None, w.cuda(), eps, dtype, groups=groups)
    close(got, pm.grouped_norm(x.to(F), w.to(F), groups, eps), tol)
    assert torch.equal(xd.cpu(), x)
    got = ops.add_rmsnorm(xd, r.cuda(), w.cuda(), eps, dtype, groups=groups)
    close(got, pm.grouped_norm((x + r).to(F), w.to(F), groups, eps), tol, "with a sum")
    close(xd, (x + r), 1e-6, "the sum itself")
    got = ops.add_rmsnorm(xd, None, w.cuda(), eps, dtype, rows=i32([T - 1, 0]), groups=groups)
    close(got, pm.grouped_norm((x + r).to(F), w.to(F), groups, eps)[[T - 1, 0]], tol, "some rows")


@pytest.mark.parametrize("groups", [1, 4])
def test_a_products_sums_are_added_before_the_norm(ops, groups):
    T, W, K = 4, 96, 64
    a, wt = rnd(T, K, seed=1).bfloat16().cuda(), rnd(W, K, seed=2, scale=0.2).bfloat16().cuda()
    x, w = rnd(T, W, seed=3), 1 + rnd(W, seed=4, scale=0.3)
    ref = x.to(F) + a.cpu().to(F) @ wt.cpu().to(F).T
    xd = x.cuda()
    pending = ops.linear(a, wt, None, out_dtype=torch.float32, accumulate_into=xd, may_defer=True)
    got = ops.add_rmsnorm(xd, pending, w.cuda(), 1e-5, torch.bfloat16, groups=groups)
    close(xd, ref, 1e-5)
    close(got, pm.grouped_norm(ref, w.to(F), groups, 1e-5), 6e-3)
    xd = x.cuda()
    got = ops.add_rmsnorm(xd, ops.linear(a, wt, None, out_dtype=torch.float32, may_defer=True), w.cuda(), 1e-5,
                          torch.bfloat16, groups=groups)
    close(got, pm.grouped_norm(ref, w.to(F), groups, 1e-5), 6e-3, "a product that nobody has taken yet")


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W,groups", [(5, 96, 4), (3, 70, 1), (4, 70, 7), (6, 2048, 4), (2, 5000, 2), (3, 4100, 5)])
def test_two_branches_are_normed_summed_and_the_next_norm_follows(ops, dtype, T, W, groups):
    from llmserve_b200.parts.base import BranchMix

    x, a, b = rnd(T, W, seed=1), rnd(T, W, seed=2, scale=20.0), rnd(T, W, seed=3, scale=0.1)
    wa, wb, w = (1 + rnd(W, seed=s, scale=0.3) for s in (4, 5, 6))
    x[:, : W // groups] *= 20
    eps = 1e-3
    ref = x.to(F) + 0.5 * (pm.unit_rms(a.to(F), eps) * wa + pm.unit_rms(b.to(F), eps) * wb)
    xd = x.cuda()
    mix = BranchMix(ops, [a.cuda(), b.cuda()], [wa.cuda(), wb.cuda()], (0.5, 0.5), eps)
    got = ops.mix_add_rmsnorm(xd, mix, w.cuda(), 1e-5, dtype, groups=groups)
    close(xd, ref, 2e-6, "the sum")
    close(got, pm.grouped_norm(ref, w.to(F), groups, 1e-5), 3e-6 if dtype == torch.float32 else 6e-3)


def test_two_products_that_lie_as_sums_are_taken_by_the_same_launch(ops):
    from llmserve_b200.parts.base import BranchMix

    T, W, K = 3, 128, 64
    h = rnd(T, K, seed=1).bfloat16().cuda()
    wts = [rnd(W, K, seed=2 + i, scale=0.2).bfloat16().cuda() for i in range(2)]
    x, wa, wb, w = rnd(T, W, seed=5), *(1 + rnd(W, seed=s, scale=0.3) for s in (6, 7, 8))
    prods = [ops.linear(h, m, None, out_dtype=torch.float32, may_defer=True) for m in wts]
    refs = [h.cpu().to(F) @ m.cpu().to(F).T for m in wts]
    xd = x.cuda()
    got = ops.mix_add_rmsnorm(xd, BranchMix(ops, prods, [wa.cuda(), wb.cuda()], (0.5, 0.5), 1e-5), w.cuda(), 1e-5,
                              torch.bfloat16, groups=2)
    ref = x.to(F) + 0.5 * (pm.unit_rms(refs[0], 1e-5) * wa + pm.unit_rms(refs[1], 1e-5) * wb)
    close(xd, ref, 1e-5)
    close(got, pm.grouped_norm(ref, w.to(F), 2, 1e-5), 6e-3)
    again = ops.linear(h, wts[0], None, out_dtype=torch.float32)  # the buffers were left zero
    close(again, refs[0], 1e-5)


# ----------------------------------------------------------------------------- chunked attention
def pages_for(n_seq, max_len, page_tokens, nk, Dp, dtype, seed=0, fill=float("nan")):
    per = -(-max_len // page_tokens)
    order = torch.randperm(n_seq * per + 3, generator=torch.Generator().manual_seed(seed))[: n_seq * per]
    tables = order.view(n_seq, per).to(torch.int32).cuda()
    k = torch.full((n_seq * per + 3, nk, page_tokens, Dp), fill, dtype=dtype).cuda()
    return tables, k, k.clone()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("nq,nk,D,Dv,rot,col0", [(4, 2, 24, 40, 8, 0), (3, 3, 18, 10, 18, 8), (8, 2, 64, 64, 64, 16),
                                                 (2, 1, 20, 12, 0, 0), (2, 2, 32, 16, 16, 4)])
def test_rotated_rows_beside_values_of_another_size(ops, dtype, nq, nk, D, Dv, rot, col0):
    q_lens, starts, page_tokens = [5, 1, 9], [0, 37, 14], 8
    b = batch(q_lens, starts, [0, 1, 2])
    T, Dp = sum(q_lens), max(D, Dv) + (-max(D, Dv)) % 16
    proj = rnd(T, col0 + (nq + nk) * D + nk * Dv + 5, seed=1)
    cos = sin = None
    if rot:
        a = torch.arange(64, dtype=F)[:, None] * (300.0 ** (-2.0 * torch.arange(rot // 2, dtype=F) / rot) / 4.0)
        cos, sin = a.cos().float().cuda(), a.sin().float().cuda()
    tables, kp, vp = pages_for(3, 48, page_tokens, nk, Dp, dtype)
    got = ops.qkv_norm_rope_write(
        proj.cuda(), col0=col0, num_heads=nq, num_kv_heads=nk, num_value_heads=nk, head_dim=D, value_dim=Dv, out_dim=Dp,
        q_weight=None, k_weight=None, eps=0.0, positions=b.positions, token_seq=b.token_seq, cos=cos, sin=sin,
        k_pages=kp, v_pages=vp, block_tables=tables, page_tokens=page_tokens, out_dtype=dtype)
    pos = b.positions.cpu().long()
    p = proj.to(F)[:, col0:]
    # the kernel pairs halves: the plain rotation of neighbours on reordered dims
    from llmserve_b200.parts.positions import neighbours_to_halves

    order = neighbours_to_halves(D, rot)
    back = torch.argsort(torch.tensor(order))
    turn = lambda x: pm.rotate_neighbours(x[..., back], pos, rot, 300.0, 4.0)[..., order]
    q, k = turn(p[:, : nq * D].view(T, nq, D)), turn(p[:, nq * D : (nq + nk) * D].view(T, nk, D))
    v = p[:, (nq + nk) * D : (nq + nk) * D + nk * Dv].view(T, nk, Dv)
    tol = 3e-6 if dtype == torch.float32 else 5e-3
    fill = lambda x: torch.nn.functional.pad(x, (0, Dp - x.shape[-1]))
    close(got.view(T, nq, Dp), fill(q), tol, "queries")
    page = tables.cpu()[b.token_seq.cpu().long(), pos // page_tokens].long().cuda()
    close(kp[page, :, (pos % page_tokens).cuda()], fill(k), tol, "keys")
    close(vp[page, :, (pos % page_tokens).cuda()], fill(v), tol, "values")


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("n_rows,splits", [(1, 1), (1, 3), (40, 0), (2, 0)])
@pytest.mark.parametrize("D,chunk,ctx", [(48, 24, 150), (48, 32, 160), (64, 37, 149), (64, 37, 112), (32, 500, 300),
                                         (16, 1, 20), (64, 16, 97)])
def test_a_planted_key_at_the_chunks_edge(ops, dtype, n_rows, splits, D, chunk, ctx):
    """One key matches the last query far better than all others: the chunk's first, the one before it (the
    last of the chunk before), the query's own and one far back. Only keys of the query's own chunk
    may take the weight, also where the chunk ends inside a page or the query is its first."""
    n_rows = min(n_rows, ctx)
    H, G, page_tokens = 4, 2, 16
    first = (ctx - 1) // chunk * chunk
    for at in sorted({first, max(first - 1, 0), ctx - 1, 0}):
        q, k, v = rnd(ctx, H, D, seed=1, scale=0.3), rnd(ctx, G, D, seed=2, scale=0.3), rnd(ctx, G, D, seed=3)
        k[at] = 0
        k[at, :, 0] = 6.0
        q[-1] = 0
        q[-1, :, 0] = 6.0
        b = batch([n_rows], [ctx - n_rows], [0])
        b.decode_splits = splits if n_rows == 1 else 0
        tables, kp, vp = pages_for(1, ctx, page_tokens, G, D, dtype, seed=3, fill=0.5)
        pos = torch.arange(ctx)
        page = tables.cpu()[0, pos // page_tokens].long().cuda()
        kp[page, :, (pos % page_tokens).cuda()] = k.to(dtype).cuda()
        vp[page, :, (pos % page_tokens).cuda()] = v.to(dtype).cuda()
        ops.check_attention_shape(D, dtype, H, G)
        plan = {n: torch.from_numpy(a).cuda() for n, a in ops.attention_plan(b.host, dtype, D).items()}
        got = ops.paged_attention(
            q[ctx - n_rows:].reshape(n_rows, H * D).to(dtype).cuda().contiguous(), num_heads=H, num_kv_heads=G, head_dim=D,
            scale=0.5, window=0, k_pages=kp, v_pages=vp, block_tables=tables, page_tokens=page_tokens, step=b, plan=plan,
            chunk=chunk)
        ref = pm.attend(q.to(F), k.to(F), v.to(F), 0.5, pm.chunk_mask(ctx, chunk))[ctx - n_rows:]
        close(got.view(n_rows, H, D), ref, 2e-5 if dtype == torch.float32 else 2e-2, f"key {at}")
        takes = (ref[-1, 0] - v[at, 0].to(F)).abs().max().item() < 0.05
        assert takes == (at >= first), at


# ----------------------------------------------------------------------------- gated delta rule
def delta_case(H, G, dk, dv, taps, T, slots, seed=1):
    C = 2 * G * dk + H * dv
    return SimpleNamespace(
        H=H, G=G, dk=dk, dv=dv, taps=taps, C=C, proj=rnd(T, 8 + C + H * dv + 2 * H + 3, seed=seed),
        conv=rnd(taps, C, seed=seed + 1, scale=0.6), A=rnd(H, seed=seed + 2), dt=rnd(H, seed=seed + 3),
        inputs=rnd(slots, max(taps - 1, 1), C, seed=seed + 4), S=rnd(slots, H, dv, dk, seed=seed + 5, scale=0.3))


def delta_run(ops, c, proj, b, inputs, S):
    kw = dict(num_heads=c.H, num_kv_heads=c.G, key_dim=c.dk, value_dim=c.dv, step=b)
    qkv, scal = ops.delta_inputs(proj.cuda(), 8, conv=c.conv.cuda(), conv_state=inputs if c.taps > 1 else None,
                                 A_log=c.A.cuda(), dt_bias=c.dt.cuda(), query_scale=c.dk ** -0.5, **kw)
    return ops.delta_rule(qkv, scal, state=S, **kw)


def delta_plain(c, proj, before, S0):
    """One sequence in float64: outputs, the last inputs, the last state (transposed as it is kept)."""
    n, H, G, dk, dv, C = proj.shape[0], c.H, c.G, c.dk, c.dv, c.C
    p = proj[:, 8:].to(F)
    x = torch.cat([torch.zeros(c.taps - 1, C, dtype=F) if before is None else before.to(F)[: c.taps - 1], p[:, :C]])
    y = pm.silu(pm.short_conv(x, c.conv.to(F).t()))[c.taps - 1 :]
    rep = lambda t: t.repeat_interleave(H // G, 1)
    q = rep(pm.unit_vector(y[:, : G * dk].view(n, G, dk))) * dk ** -0.5
    k = rep(pm.unit_vector(y[:, G * dk : 2 * G * dk].view(n, G, dk)))
    b0 = C + H * dv
    o, S = pm.delta_rule(q, k, y[:, 2 * G * dk :].view(n, H, dv), torch.sigmoid(p[:, b0 : b0 + H]),
                         pm.decay(p[:, b0 + H : b0 + 2 * H], c.A.to(F), c.dt.to(F)),
                         None if S0 is None else S0.to(F).transpose(1, 2))
    return o.reshape(n, H * dv), x[x.shape[0] - (c.taps - 1) :], S.transpose(1, 2)


SIZES = [(1, 1, 16, 520, 2), (4, 2, 64, 32, 4), (3, 3, 20, 12, 3), (2, 1, 128, 128, 4), (1, 1, 256, 40, 2), (5, 5, 16, 24, 1), (2, 2, 48, 72, 5),
         (4, 4, 12, 10, 4), (3, 1, 7, 9, 4), (2, 1, 132, 136, 4), (1, 1, 64, 256, 3)]


@pytest.mark.parametrize("sizes", SIZES)
def test_delta_rule_in_chunks_portions_and_single_tokens(ops, sizes):
    """A ragged batch: long portions that run as chunks side by side (from zero and from a state), short
    ones, first tokens on slots that hold garbage, single tokens behind a state; then every
    sequence goes on one token at a time."""
    L = int(ops.ext.delta_rule_chunk())
    q_lens, starts, slots = [3 * L + 8, 9, 1, 1, L + 1, 2, 2 * L, L], [0, 5, 0, 30, 11, 0, L, 3], [3, 0, 4, 1, 2, 6, 5, 8]
    c = delta_case(*sizes, T=sum(q_lens), slots=10)
    b = batch(q_lens, starts, slots)
    inputs, S = c.inputs.cuda(), c.S.cuda()
    got = delta_run(ops, c, c.proj, b, inputs, S)
    at, kept = 0, []
    for n, s0, slot in zip(q_lens, starts, slots):
        ref, xs, Sn = delta_plain(c, c.proj[at : at + n], c.inputs[slot] if s0 else None, c.S[slot] if s0 else None)
        close(got[at : at + n], ref, 3e-6, f"sequence of {n} from {s0}")
        close(S[slot], Sn, 3e-6, "the state left behind")
        if c.taps > 1:
            close(inputs[slot], xs, 1e-7, "the inputs left behind")
        kept.append((xs, Sn))
        at += n
    assert torch.equal(S[[7, 9]].cpu(), c.S[[7, 9]]), "a slot that no sequence uses was touched"
    assert torch.equal(inputs[[7, 9]].cpu(), c.inputs[[7, 9]])
    for k in range(6):
        nb = batch([1] * len(slots), [s + n + k for s, n in zip(starts, q_lens)], slots)
        p1 = rnd(len(slots), c.proj.shape[1], seed=50 + k)
        got = delta_run(ops, c, p1, nb, inputs, S)
        for i in range(len(slots)):
            ref, xs, Sn = delta_plain(c, p1[i : i + 1], *kept[i])
            close(got[i : i + 1], ref, 5e-6, f"single token {k} of sequence {i}")
            kept[i] = (xs, Sn)


@pytest.mark.parametrize("cuts", [[300], [1] * 12 + [288], [2] * 20 + [260], [63, 64, 65, 66, 42], [129, 2, 1, 168], [3, 297]])
def test_delta_rule_does_not_depend_on_the_cut(ops, cuts):
    n = sum(cuts)
    c = delta_case(3, 1, 24, 40, 4, T=n, slots=2)
    inputs, S = c.inputs.cuda(), c.S.cuda()
    outs, at = [], 0
    for m in cuts:
        outs.append(delta_run(ops, c, c.proj[at : at + m], batch([m], [at], [1]), inputs, S))
        at += m
    ref, xs, Sn = delta_plain(c, c.proj, None, None)
    close(torch.cat(outs), ref, 3e-6)
    close(S[1], Sn, 3e-6)
    close(inputs[1], xs, 1e-7)


@pytest.mark.parametrize("gap", [1, 5, 63, 64, 65, 150])
def test_a_key_is_found_again_and_a_second_write_replaces_the_first(ops, gap):
    """Without decay and with full steps a key's value is read back exactly however many other keys came
    between, across chunk borders too; writing the key again replaces the value; a head that
    decays at once forgets it."""
    H, G, dk, dv = 2, 1, 32, 16
    n = 2 * gap + 3
    qkv = torch.zeros(n, 2 * G * dk + H * dv)
    qkv[:, 0] = 1.0  # every query asks for key 0
    for t in range(n):  # other keys: all but direction 0
        qkv[t, dk + 1 + t % (dk - 1)] = 1.0
    for t, val in ((0, 1.0), (gap + 1, 5.0)):
        qkv[t, dk : 2 * dk] = 0
        qkv[t, dk] = 1.0
        qkv[t, 2 * dk :] = val
    scal = torch.zeros(n, H, 4)
    scal[:, 0, 0], scal[:, 1, 0] = 1.0, 1e-30  # the decays of the two heads
    scal[:, :, 1] = 1.0
    scal[:, :, 2] = (qkv[:, :dk] * qkv[:, dk : 2 * dk]).sum(1, keepdim=True)
    S = rnd(1, H, dv, dk).cuda()
    out = ops.delta_rule(qkv.cuda(), scal.cuda().contiguous(), num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, state=S,
                         step=batch([n], [0], [0])).cpu().view(n, H, dv)
    close(out[0], torch.ones(H, dv), 1e-6)
    close(out[1 : gap + 1, 0], torch.ones(gap, dv), 1e-5, "still there")
    close(out[gap + 1 :, 0], torch.full((gap + 2, dv), 5.0), 1e-5, "replaced")
    close(out[1 : gap + 1, 1], torch.zeros(gap, dv), 1e-6, "forgotten")


# ----------------------------------------------------------------------------- feed-forward
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,K,N", [(1, 64, 96), (5, 70, 50), (3, 128, 2052), (40, 64, 112), (33, 96, 9000), (2, 64, 16384),
                                   (2, 64, 20000)])
def test_polynomial_of_norms(ops, dtype, T, K, N):
    h, w = rnd(T, K, seed=1).to(dtype), rnd(N, K, seed=2, scale=0.2).to(dtype)
    coef = torch.tensor([0.7, -0.4, 0.3, 0.25])
    got = ops.poly_norm_linear(h.cuda(), w.cuda(), coef.cuda(), 1e-5, dtype)
    z = h.to(F) @ w.to(F).T
    close(got, pm.poly_norm(z, coef.to(F), 1e-5), 1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,I", [(1, 64), (5, 50), (40, 96), (300, 1024)])
def test_clamped_gate(ops, dtype, T, I):
    gu = rnd(T, 2 * I, seed=1, scale=2.0)
    for limit in (0.5, 1.7):
        got = ops.silu_mul(gu.cuda(), out_dtype=dtype, activation="clamped_glu", limit=limit)
        close(got, pm.clamped_glu(gu[:, :I].to(F), gu[:, I:].to(F), limit), 2e-6 if dtype == torch.float32 else 8e-3)
    gu[:, :I], gu[:, I:] = -40.0, 40.0  # the gate is cut from above only, the other from both sides
    got = ops.silu_mul(gu.cuda(), out_dtype=dtype, activation="clamped_glu", limit=1.5)
    close(got, pm.clamped_glu(gu[:, :I].to(F), gu[:, I:].to(F), 1.5), 1e-6)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W,E,top,groups,keep", [(7, 64, 6, 2, 3, 1), (5, 70, 8, 3, 4, 2), (3, 96, 14, 4, 2, 1),
                                                   (40, 128, 40, 5, 8, 3), (4, 32, 5, 5, 1, 1), (6, 48, 64, 1, 64, 1)])
def test_router_with_groups_and_a_correction(ops, dtype, T, W, E, top, groups, keep):
    h, router = rnd(T, W, seed=1).to(dtype), rnd(E + 1, W, seed=2, scale=0.3)
    corr = rnd(E, seed=3) - 1.5  # most choice scores are negative: an excluded group must not count as 0
    idx, wts, gate = ops.moe_route(h.cuda(), router.cuda(), E, top, True, bias=corr.cuda(), weights="softmax_of_all",
                                   groups=groups, keep=keep, scale=1.7)
    z = h.to(F) @ router.to(F).T
    ri, rw = pm.choose(z[:, :E], corr.to(F), top, groups, keep, 1.7)
    assert torch.equal(idx.cpu().long(), ri)
    close(wts, rw, 1e-5)
    close(gate, torch.sigmoid(z[:, E]), 1e-5)
    # without the correction others are chosen here and there, with the same scores as weights
    plain = pm.choose(z[:, :E], torch.zeros(E, dtype=F), top, groups, keep, 1.7)[0]
    if top < E and E < 40:
        assert not torch.equal(plain, ri)


def test_router_ties_go_to_the_lower_index(ops):
    idx, wts, _ = ops.moe_route(torch.ones(2, 16).cuda(), torch.ones(9, 16).cuda(), 9, 2, False,
                                weights="softmax_of_all", groups=3, keep=1, scale=2.0)
    assert idx.cpu().tolist() == [[0, 1], [0, 1]]
    close(wts, torch.ones(2, 2), 1e-6)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W,E,ident,top,ff,shared,groups,keep", [
    (1, 64, 4, 2, 2, 32, 48, 2, 1), (9, 96, 6, 0, 3, 24, 0, 1, 1), (40, 64, 3, 5, 4, 16, 32, 4, 3),
    (7, 70, 5, 1, 2, 18, 10, 3, 2), (600, 128, 6, 2, 2, 64, 64, 2, 1), (50, 64, 1, 3, 2, 16, 0, 2, 1)])
def test_experts_with_identity_experts_against_the_plain_sum(ops, dtype, T, W, E, ident, top, ff, shared, groups, keep):
    """Every kernel of the experts' products (few choices, tiles, tcgen05 tiles, CUDA cores), with choices
    that have no row in the sorted order, also where most or all choices of the step are such."""
    from llmserve_b200.parts.base import BuildEnv
    from llmserve_b200.parts.moe import RoutedExperts, RoutedExpertsSpec

    env = BuildEnv(ops=ops, dtype=dtype, device=torch.device("cuda"), max_positions=8, branch_dtype=torch.float32)
    part = RoutedExperts(RoutedExpertsSpec(
        W, E, top, ff, shared, activation="clamped_glu", router_weights="softmax_of_all", weight_on="output", correction=True,
        groups=groups, keep_groups=keep, router_scale=1.5, identity_experts=ident, limit=0.9, shared_limit=0.6), env)
    params, w = {}, {}
    for k, (name, decl) in enumerate(part.param_decls().items()):
        t = rnd(*decl.shape, seed=k, scale=1.0 if "router" in name else 0.3)
        params[name] = (t.to(dtype) if decl.role == "matrix" else t).cuda().contiguous()
    for e in range(E):
        gu = params["experts.gate_up.weight"].view(E, 2 * ff, W)[e].cpu().to(F)
        w[f"e{e}.gate"], w[f"e{e}.up"] = gu[:ff], gu[ff:]
        w[f"e{e}.down"] = params["experts.down.weight"].view(E, W, ff)[e].cpu().to(F)
    w["router"], w["correction"] = params["router.weight"][: E + ident].cpu().to(F), params["router.correction"].cpu().to(F)
    mlp = {"router": {"experts": E, "top": top, "groups": {"count": groups, "keep": keep}, "identity": ident, "scale": 1.5},
           "expert": {"ff": ff, "limit": 0.9}}
    if shared:
        gu = params["shared.gate_up.weight"].cpu().to(F)
        w["shared.gate"], w["shared.up"] = gu[:shared], gu[shared:]
        w["shared.down"], w["shared.sg"] = params["shared.down.weight"].cpu().to(F), params["router.weight"][E + ident:].cpu().to(F)
        mlp["shared"] = {"ff": shared, "limit": 0.6}
    part.bind(params)
    h = rnd(T, W, seed=99).to(dtype)
    x = rnd(T, W, seed=98)
    ref = x.to(F) + pm.moe(h.to(F), w, "", mlp)
    xd = x.cuda()
    assert part.forward(h.cuda(), None, residual=xd) is None
    close(xd, ref, 1e-5 if dtype == torch.float32 else 1e-2)
    if ident:
        close(part.forward(h.cuda(), None), ref - x.to(F), 2e-5 if dtype == torch.float32 else 1e-2, "returned")
        only = params["router.correction"].clone()
        only[:E] -= 10.0  # real experts are chosen only where no identity expert is left
        part.correction = only
        w["correction"] = only.cpu().to(F)
        xd = x.cuda()
        part.forward(h.cuda(), None, residual=xd)
        close(xd, x.to(F) + pm.moe(h.to(F), w, "", mlp), 1e-5 if dtype == torch.float32 else 1e-2, "identity experts first")
    ops.check_kernel_errors()


# ----------------------------------------------------------------------------- the model
def gpu_runner(folder, name, num_pages, dtype, max_num_seqs=4, max_len=512):
    from llmserve_b200.engine.runner import ModelRunner, load_model
    from llmserve_b200.ops import get_ops

    _, _, model = load_model(folder, dtype, "cuda", get_ops("cuda"), max_len)
    return ModelRunner(model, page_tokens=MIBERAX_TINY[name]["page_tokens"], num_pages=num_pages,
                       max_model_len=max_len, max_num_seqs=max_num_seqs, max_num_batched_tokens=max_len)


LENGTHS = {"M1": [5, 70, 1, 33, 49, 190, 2], "M2": [2, 40, 9, 64, 17, 100], "M3": [3, 150, 18, 77, 230]}
TOL = {"float32": (3e-4, 2e-5), "bfloat16": (0.0, 0.03)}  # (absolute, relative to the largest logit)


@pytest.fixture(scope="module")
def expected(miberax_dirs):
    out = {}
    for name in NAMES:
        reqs = traces.make_requests(LENGTHS[name], MIBERAX_TINY[name]["config"]["vocab"], seed=5)
        out[name] = (reqs, {r: pm.model_logits(miberax_dirs[name], t) for r, t in reqs.items()})
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("mode", ["whole", "decode_tail", "portions", "mixed"])
def test_every_way_of_cutting_matches_plain(miberax_dirs, expected, name, mode, dtype):
    reqs, exp = expected[name]
    runner = gpu_runner(miberax_dirs[name], name, traces.tokens_needed(reqs) // MIBERAX_TINY[name]["page_tokens"], dtype)
    got = traces.replay(runner, getattr(traces, mode)(reqs))
    atol, rtol = TOL[dtype]
    traces.compare(got, exp, atol=atol, rtol=rtol)
    assert runner.manager.usage() == 0.0
    runner.check_kernels()


@pytest.mark.parametrize("name", NAMES)
def test_layers_one_by_one_in_float32(miberax_dirs, name):
    folder = miberax_dirs[name]
    tokens = traces.make_requests([150], MIBERAX_TINY[name]["config"]["vocab"], seed=2)["r0"]
    cfg, w = pm.load(folder)
    _, after = pm.forward(tokens, w, cfg, return_layers=True)
    runner = gpu_runner(folder, name, 20, "float32")
    seen = []
    for block in runner.model.blocks:
        inner = block.forward

        def spy(x, pending, step, cache, inner=inner):
            x, pending = inner(x, pending, step, cache)
            pending = pending.resolve() if hasattr(pending, "resolve") else pending
            if pending is not None:
                x = x + pending
            seen.append(x.clone())
            return x, None

        block.forward = spy
    from llmserve_b200.engine.batch import StepEntry

    runner.run([StepEntry("a", tokens, [0])])
    assert len(seen) == len(cfg["layers"])
    for i, x in enumerate(seen):
        close(x, after[i], 2e-5, f"after layer {i}")


def test_float32_logits_do_not_depend_on_the_cut(miberax_dirs, expected):
    reqs, _ = expected["M1"]
    pool = traces.tokens_needed(reqs) // 16
    a = traces.replay(gpu_runner(miberax_dirs["M1"], "M1", pool, "float32"), traces.whole(reqs))
    b = traces.replay(gpu_runner(miberax_dirs["M1"], "M1", pool, "float32"), traces.mixed(reqs, seed=4))
    scale = max(v.abs().max().item() for v in a.values())
    assert max((a[k] - b[k]).abs().max().item() for k in a) <= 2e-5 * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_from_the_first_token_on_few_pages(miberax_dirs, dtype):
    """300 tokens one by one from position 0 on a seventh of the pages they would need without chunks."""
    reqs = traces.make_requests([300], 131, seed=21)
    exp = {r: pm.model_logits(miberax_dirs["M2"], t) for r, t in reqs.items()}
    runner = gpu_runner(miberax_dirs["M2"], "M2", 6, dtype)
    got = traces.replay(runner, traces.decode_tail(reqs, tail=300))
    atol, rtol = TOL[dtype]
    traces.compare(got, exp, atol=atol, rtol=rtol)


def test_slots_and_pages_used_again(miberax_dirs):
    """One state slot and just enough pages: every request runs on what the one before it left."""
    reqs = traces.make_requests([40, 37, 64, 3, 150], 163, seed=8)
    exp = {r: pm.model_logits(miberax_dirs["M1"], t) for r, t in reqs.items()}
    runner = gpu_runner(miberax_dirs["M1"], "M1", 10, "float32", max_num_seqs=1)
    traces.compare(traces.replay(runner, traces.portions(reqs)), exp, atol=3e-4, rtol=2e-5)


@pytest.mark.parametrize("name", ["M1", "M3"])
def test_steps_that_want_some_rows_or_none(miberax_dirs, name):
    wanted_subsets(lambda: gpu_runner(miberax_dirs[name], name, 16, "float32"), miberax_dirs[name],
                   MIBERAX_TINY[name]["config"]["vocab"], 3e-4)
    wanted_subsets(lambda: gpu_runner(miberax_dirs[name], name, 16, "bfloat16"), miberax_dirs[name],
                   MIBERAX_TINY[name]["config"]["vocab"], 0.0, 0.06)


# ----------------------------------------------------------------------------- generation
PROMPTS = [[5, 9, 90, 31, 7], list(range(40, 57)), [3] * 33, [90, 2], list(range(90))]


def llm(folder, name, dtype, **kw):
    from llmserve_b200 import LLM

    d = dict(dtype=dtype, block_size=MIBERAX_TINY[name]["page_tokens"], num_kv_blocks=64, max_model_len=256,
             max_num_seqs=8)
    d.update(kw)
    return LLM(str(folder), **d)


def greedy(n):
    from llmserve_b200 import SamplingParams

    return SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True)


@pytest.mark.parametrize("name", ["M1", "M2"])
@pytest.mark.parametrize("kw", [dict(cuda_graphs=False), dict(cuda_graphs=True),
                                dict(cuda_graphs=True, max_num_batched_tokens=24),
                                dict(cuda_graphs=True, num_kv_blocks=14, max_num_batched_tokens=16)])
def test_greedy_float32_equals_plain_greedy(miberax_dirs, name, kw):
    """Through the entry point: the scheduler's batches, captured steps (single tokens and padded
    steps with portions), preemption by recomputation."""
    m = llm(miberax_dirs[name], name, "float32", **kw)
    outs = m.generate(PROMPTS, greedy(12))
    for o, p in zip(outs, PROMPTS):
        assert o.outputs[0].token_ids == pm.greedy(miberax_dirs[name], p, 12), (kw, p)


def test_greedy_bfloat16_picks_tokens_the_plain_model_also_ranks_first(miberax_dirs):
    outs = llm(miberax_dirs["M1"], "M1", "bfloat16", cuda_graphs=True).generate(PROMPTS, greedy(10))
    for o, p in zip(outs, PROMPTS):
        gen = o.outputs[0].token_ids
        logits = pm.model_logits(miberax_dirs["M1"], p + gen)[len(p) - 1 : -1]
        for t, row in zip(gen, logits):
            assert float(row.max() - row[t]) <= 0.03 * float(row.abs().max())
