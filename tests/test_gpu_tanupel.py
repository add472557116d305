"""The Tanupel parts on the GPU: each kernel against the plain float64 function of its mechanism,
then the model through the step function and through generation, against the plain model."""

from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_tanupel as pt
import traces
from conftest import TANUPEL_TINY
from test_tanupel_cpu import wanted_subsets

pytestmark = pytest.mark.gpu

F = torch.float64
NAMES = sorted(TANUPEL_TINY)
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


# ----------------------------------------------------------------------------- embedding, sums, norm
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("W", [64, 70, 2056])
def test_embedding_times_a_constant(ops, dtype, W):
    table = rnd(11, W, seed=1).to(dtype)
    ids = [3, 0, 10, 3]
    close(ops.embedding(i32(ids), table.cuda(), 2.5), table.double()[ids] * 2.5, 1e-6)
    assert torch.equal(ops.embedding(i32(ids), table.cuda()).cpu(), table.float()[ids])


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W", [(1, 64), (5, 70), (3, 2048), (2, 4099), (2, 16388), (2, 20000), (300, 64), (260, 2048)])
@pytest.mark.parametrize("n,with_row", [(0, True), (1, False), (3, True), (4, False), (6, True)])
def test_several_results_a_vector_and_the_next_norm(ops, dtype, T, W, n, with_row):
    x, row, w = rnd(T, W, seed=1), rnd(W, seed=2), rnd(W, seed=3, scale=0.4)
    ys = [rnd(T, W, seed=10 + i, scale=1.0 + i) for i in range(n)]
    cs = [0.5, -1.25, 3.0, 0.1, 2.0, -0.7][:n]
    ref = x.to(F) + sum(c * y.to(F) for c, y in zip(cs, ys)) + (row.to(F) if with_row else 0.0)
    items = [(c, y.cuda()) for c, y in zip(cs, ys)]
    r = row.cuda() if with_row else None
    xd = x.cuda()
    got = ops.sum_add_rmsnorm(xd, items, r, (1 + w).cuda(), 0.01, dtype)
    close(xd, ref, 2e-6, "the sum")
    close(got, pt.offset_norm(ref, w.to(F), 0.01), 3e-6 if dtype == torch.float32 else 6e-3, "the norm")
    xd = x.cuda()
    assert ops.sum_add(xd, items, r) is None
    close(xd, ref, 2e-6, "the sum alone")


def test_products_that_lie_as_sums_are_scaled_and_taken_by_the_same_launch(ops):
    T, W, K = 3, 128, 64
    h = rnd(T, K, seed=1).bfloat16().cuda()
    wts = [rnd(W, K, seed=2 + i, scale=0.2).bfloat16().cuda() for i in range(3)]
    x, y, w = rnd(T, W, seed=5), rnd(T, W, seed=6), rnd(W, seed=7, scale=0.3)
    xd = x.cuda()
    prods = [ops.linear(h, m, None, out_dtype=torch.float32, accumulate_into=xd, coefficient=c, may_defer=True)
             for m, c in zip(wts, (0.3, -2.0, 1.0))]
    assert all(hasattr(p, "resolve") for p in prods) and torch.equal(xd.cpu(), x), "nothing is added before the norm"
    refs = [h.cpu().to(F) @ m.cpu().to(F).T for m in wts]
    got = ops.sum_add_rmsnorm(xd, list(zip((0.3, -2.0, 1.0), prods)) + [(0.5, y.cuda())], None, (1 + w).cuda(), 1e-5,
                              torch.bfloat16)
    ref = x.to(F) + 0.3 * refs[0] - 2.0 * refs[1] + refs[2] + 0.5 * y.to(F)
    close(xd, ref, 1e-5)
    close(got, pt.offset_norm(ref, w.to(F), 1e-5), 6e-3)
    close(ops.linear(h, wts[0], None, out_dtype=torch.float32), refs[0], 1e-5, "the buffers were left zero")


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T", [2, 33, 200])
def test_a_product_is_added_times_a_constant(ops, dtype, T):
    from llmserve_b200.parts.base import PendingAdds, add_projected

    a, w, x = rnd(T, 96, seed=1).to(dtype), rnd(80, 96, seed=2, scale=0.2).to(dtype), rnd(T, 80, seed=3)
    xd = x.cuda()
    items = add_projected(ops, a.cuda(), w.cuda(), None, xd, -0.35)
    PendingAdds(ops, xd, items).resolve()
    close(xd, x.to(F) - 0.35 * (a.to(F) @ w.to(F).T), 1e-5)


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,I,col0", [(1, 64, 8), (5, 50, 24), (40, 1028, 16)])
def test_gate_from_columns_of_a_wider_product(ops, dtype, T, I, col0):
    proj = rnd(T, col0 + 2 * I + 12 + (-2 * I) % 4, seed=1, scale=2.0)
    got = ops.silu_mul(proj.cuda(), out_dtype=dtype, columns=(col0, 2 * I))
    g, u = proj[:, col0 : col0 + I].to(F), proj[:, col0 + I : col0 + 2 * I].to(F)
    close(got, pt.silu(g) * u, 2e-6 if dtype == torch.float32 else 8e-3)


@pytest.mark.parametrize("T", [3, 40])
def test_both_sublayers_share_one_product_where_rows_are_few(tanupel_dirs, ops, T):
    """A dense layer: with few bfloat16 rows one product serves the mixer and the feed-forward, with many each has its
    own; the matrices are views of one."""
    from llmserve_b200.engine.batch import StepEntry

    runner = gpu_runner(tanupel_dirs["T3"], "T3", 20, "bfloat16")
    block = runner.model.blocks[0]
    w = block.shared_weight
    assert w is not None and w.data_ptr() == block.mixer.shared_weight.data_ptr() and block.ff_column % 8 == 0
    assert block.feed_forward.gate_up_weight.data_ptr() == w[block.ff_column].data_ptr()
    assert runner.model.blocks[1].shared_weight is None  # routed experts start from the rows themselves
    calls = []
    inner = ops.linear
    ops.linear = lambda a, m, *r, **k: (calls.append(m.shape[0]), inner(a, m, *r, **k))[1]
    try:
        runner.run([StepEntry("a", list(range(T)), [0])])
    finally:
        ops.linear = inner
    assert (w.shape[0] in calls) == (T == 3)


# ----------------------------------------------------------------------------- attention with a soft cap
def pages_for(n_seq, max_len, page_tokens, nk, Dp, dtype, seed=0, fill=float("nan")):
    per = -(-max_len // page_tokens)
    order = torch.randperm(n_seq * per + 3, generator=torch.Generator().manual_seed(seed))[: n_seq * per]
    tables = order.view(n_seq, per).to(torch.int32).cuda()
    k = torch.full((n_seq * per + 3, nk, page_tokens, Dp), fill, dtype=dtype).cuda()
    return tables, k, k.clone()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("kernel", [0, 1, 2, 3])
@pytest.mark.parametrize("H,G,D", [(4, 2, 64), (12, 1, 64), (3, 3, 128), (4, 1, 48), (2, 2, 144)])
def test_soft_capped_scores_on_every_kernel(ops, dtype, kernel, H, G, D):
    """Portions and single tokens in one batch, contexts that end inside pages. Two planted keys score far beyond the
    cap: without it the softmax would give one of them everything, with it both count alike."""
    if dtype == torch.float32 and kernel > 1:
        pytest.skip("one kernel family in float32")
    cap, scale, page_tokens = 3.0, 0.2, 16
    q_lens, starts = [70, 1, 1, 40, 1], [61, 200, 15, 0, 0]
    b = batch(q_lens, starts, range(5))
    tables, kp, vp = pages_for(5, 210, page_tokens, G, D, dtype, seed=3, fill=0.5)
    ops.check_attention_shape(D, dtype, H, G)
    before, ops.attention_kernel = ops.attention_kernel, kernel
    try:
        refs, rows = [], []
        for s, (n, at) in enumerate(zip(q_lens, starts)):
            ctx = at + n
            q, k, v = (rnd(ctx, m, D, seed=7 * s + i, scale=sc) for i, (m, sc) in enumerate(((H, 0.6), (G, 0.6), (G, 1.0))))
            for p, size in ((ctx // 3, 9.0), (ctx // 2, 14.0)):
                k[p] = 0
                k[p, :, 0] = size
            q[:, :, 0] = 5.0
            q, k, v = (t.to(dtype) for t in (q, k, v))
            pos = torch.arange(ctx)
            page = tables.cpu()[s, pos // page_tokens].long().cuda()
            kp[page, :, (pos % page_tokens).cuda()] = k.cuda()
            vp[page, :, (pos % page_tokens).cuda()] = v.cuda()
            refs.append(pt.attend(q.to(F), k.to(F), v.to(F), scale, cap)[at:])
            rows.append(q[at:])
        plan = {n: torch.from_numpy(a).cuda() for n, a in ops.attention_plan(b.host, dtype, D).items()}
        for splits in (0, 1, 3):
            b.decode_splits = splits
            got = ops.paged_attention(
                torch.cat(rows).reshape(-1, H * D).cuda().contiguous(), num_heads=H, num_kv_heads=G, head_dim=D, scale=scale,
                window=0, k_pages=kp, v_pages=vp, block_tables=tables, page_tokens=page_tokens, step=b, plan=plan, softcap=cap)
            close(got.view(-1, H, D), torch.cat(refs), 5e-6 if dtype == torch.float32 else 2e-2, f"splits {splits}")
    finally:
        ops.attention_kernel = before
    ops.check_kernel_errors()


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("n_rows,splits", [(1, 1), (1, 3), (40, 0), (2, 0)])
@pytest.mark.parametrize("D,ctx", [(48, 150), (64, 161), (128, 97)])
def test_a_planted_key_takes_the_weight_wherever_it_stands(ops, dtype, n_rows, splits, D, ctx):
    """The sequence's first key, a page's last and the next one's first, the query's own, one before it: under a cap
    that leaves it far ahead of the others, the last query's output is that key's value. The key one behind the
    query lies in the page too and must not count."""
    H, G, page_tokens = 4, 2, 16
    for at in (0, 15, 16, 79, ctx - 2, ctx - 1, ctx):
        q, k, v = rnd(ctx, H, D, seed=1, scale=0.3), rnd(ctx + 1, G, D, seed=2, scale=0.3), rnd(ctx + 1, G, D, seed=3)
        k[at] = 0
        k[at, :, 0] = 6.0
        q[-1] = 0
        q[-1, :, 0] = 6.0
        b = batch([n_rows], [ctx - n_rows], [0])
        b.decode_splits = splits if n_rows == 1 else 0
        tables, kp, vp = pages_for(1, ctx + 1, page_tokens, G, D, dtype, seed=3, fill=0.5)
        pos = torch.arange(ctx + 1)
        page = tables.cpu()[0, pos // page_tokens].long().cuda()
        kp[page, :, (pos % page_tokens).cuda()] = k.to(dtype).cuda()
        vp[page, :, (pos % page_tokens).cuda()] = v.to(dtype).cuda()
        ops.check_attention_shape(D, dtype, H, G)
        plan = {n: torch.from_numpy(a).cuda() for n, a in ops.attention_plan(b.host, dtype, D).items()}
        got = ops.paged_attention(
            q[ctx - n_rows:].reshape(n_rows, H * D).to(dtype).cuda().contiguous(), num_heads=H, num_kv_heads=G, head_dim=D,
            scale=0.5, window=0, k_pages=kp, v_pages=vp, block_tables=tables, page_tokens=page_tokens, step=b, plan=plan,
            softcap=15.0)
        ref = pt.attend(q.to(F), k[:ctx].to(F), v[:ctx].to(F), 0.5, 15.0)[ctx - n_rows:]
        close(got.view(n_rows, H, D), ref, 2e-5 if dtype == torch.float32 else 2e-2, f"key {at}")
        if at < ctx:
            assert (ref[-1, 0] - v[at, 0].to(F)).abs().max().item() < 0.05, at


def test_a_soft_cap_is_exact_from_the_smallest_to_the_largest_scores(ops):
    """One key per score: the weights against a neutral second key give the capped score back."""
    D, page_tokens, cap = 16, 16, 30.0
    scores = torch.tensor([0.0, 1e-6, -1e-3, 0.5, -5.0, 29.0, 60.0, -200.0, 4e4, -4e4], dtype=F)
    for sc in scores:
        tables, kp, vp = pages_for(1, 2, page_tokens, 1, D, torch.float32, fill=0.0)
        page = int(tables[0, 0])
        kp[page, 0, 0, 0] = float(sc)
        vp[page, 0, 0, 0] = 1.0
        q = torch.zeros(1, D)
        q[0, 0] = 1.0
        b = batch([1], [1], [0])
        plan = {n: torch.from_numpy(a).cuda() for n, a in ops.attention_plan(b.host, torch.float32, D).items()}
        got = ops.paged_attention(q.cuda(), num_heads=1, num_kv_heads=1, head_dim=D, scale=1.0, window=0, k_pages=kp, v_pages=vp,
                                  block_tables=tables, page_tokens=page_tokens, step=b, plan=plan, softcap=cap)[0, 0].item()
        assert abs(got - torch.sigmoid(cap * torch.tanh(sc / cap)).item()) <= 2e-6, sc


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("nq,nk,D,Dv,rot", [(6, 2, 24, 40, 8), (3, 3, 18, 10, 18), (4, 1, 64, 64, 0), (8, 8, 96, 32, 24)])
def test_rows_are_normed_whole_then_turned(ops, dtype, nq, nk, D, Dv, rot):
    q_lens, starts, page_tokens, col0 = [5, 1, 9], [0, 37, 14], 8, 16
    b = batch(q_lens, starts, [0, 1, 2])
    T, Dp = sum(q_lens), max(D, Dv) + (-max(D, Dv)) % 16
    proj = rnd(T, col0 + (nq + nk) * D + nk * Dv + 5, seed=1)
    proj[:, col0 : col0 + D] *= 20  # one head much larger: a norm head by head would show
    qw, kw = 1 + rnd(nq * D, seed=2, scale=0.3), 1 + rnd(nk * D, seed=3, scale=0.3)
    r = {"base": 300.0, "dims": rot, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 60}}
    cos = sin = None
    if rot:
        a = torch.arange(64, dtype=F)[:, None] * pt.frequencies(r)[None]
        cos, sin = a.cos().float().cuda(), a.sin().float().cuda()
    tables, kp, vp = pages_for(3, 48, page_tokens, nk, Dp, dtype)
    got = ops.qkv_norm_rope_write(
        proj.cuda(), col0=col0, num_heads=nq, num_kv_heads=nk, num_value_heads=nk, head_dim=D, value_dim=Dv, out_dim=Dp,
        q_weight=qw.cuda(), k_weight=kw.cuda(), eps=0.01, positions=b.positions, token_seq=b.token_seq, cos=cos, sin=sin,
        k_pages=kp, v_pages=vp, block_tables=tables, page_tokens=page_tokens, out_dtype=dtype)
    pos, p = b.positions.cpu().long(), proj.to(F)[:, col0:]
    q = pt.rotate_halves((pt.unit_rms(p[:, : nq * D], 0.01) * qw).view(T, nq, D), pos, r)
    k = pt.rotate_halves((pt.unit_rms(p[:, nq * D : (nq + nk) * D], 0.01) * kw).view(T, nk, D), pos, r)
    v = p[:, (nq + nk) * D : (nq + nk) * D + nk * Dv].view(T, nk, Dv)
    tol = 3e-6 if dtype == torch.float32 else 5e-3
    fill = lambda x: torch.nn.functional.pad(x, (0, Dp - x.shape[-1]))
    close(got.view(T, nq, Dp), fill(q), tol, "queries")
    page = tables.cpu()[b.token_seq.cpu().long(), pos // page_tokens].long().cuda()
    close(kp[page, :, (pos % page_tokens).cuda()], fill(k), tol, "keys")
    close(vp[page, :, (pos % page_tokens).cuda()], fill(v), tol, "values")


# ----------------------------------------------------------------------------- delta rule, decays per channel
@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T", [1, 7, 32, 33, 130])
@pytest.mark.parametrize("N,K,col0", [(48, 8, 16), (70, 24, 8), (256, 128, 0), (130, 264, 24)])
def test_low_rank_products_of_both_halves(ops, dtype, T, N, K, col0):
    proj, w = rnd(T, col0 + 2 * K + 8, seed=1), rnd(2, N, K, seed=2, scale=0.2).to(dtype)
    got = ops.inner_linear(proj.cuda(), col0, w.cuda(), dtype)
    low = proj[:, col0 : col0 + 2 * K].view(T, 2, K).to(F)
    ref = torch.einsum("thk,hnk->thn", low, w.to(F)).reshape(T, 2 * N)
    close(got, ref, 1e-5 if dtype == torch.float32 or T <= 32 else 6e-3)


def delta_case(H, G, dk, dv, taps, T, slots, seed=1, decay="mixed"):
    C = 2 * G * dk + H * dv
    c = SimpleNamespace(
        H=H, G=G, dk=dk, dv=dv, taps=taps, C=C, proj=rnd(T, 8 + C + H + 5 + (-(C + H + 13)) % 4, seed=seed),
        conv=rnd(taps, C, seed=seed + 1, scale=0.6), A=rnd(H, seed=seed + 2), dt=rnd(H * dk, seed=seed + 3, scale=2.0),
        z=rnd(T, H * dk + 8, seed=seed + 6, scale=2.0),
        inputs=rnd(slots, max(taps - 1, 1), C, seed=seed + 4), S=rnd(slots, H, dv, dk, seed=seed + 5, scale=0.3))
    if decay == "slow":
        c.dt -= 8
    elif decay == "fast":  # products of a chunk's decays leave the range of float32
        c.dt += 6
        c.A += 2
    elif decay == "both":  # every other channel
        c.dt[::2] -= 8
        c.dt[1::2] += 8
    return c


def delta_run(ops, c, proj, z, b, inputs, S):
    kw = dict(num_heads=c.H, num_kv_heads=c.G, key_dim=c.dk, value_dim=c.dv, step=b)
    qkv, scal, decay = ops.delta_inputs(proj.cuda(), 8, conv=c.conv.cuda(), conv_state=inputs if c.taps > 1 else None,
                                        A_log=c.A.cuda(), dt_bias=c.dt.cuda(), query_scale=c.dk ** -0.5, decay_logits=z.cuda(), **kw)
    return ops.delta_rule(qkv, scal, state=S, decay=decay, **kw)


def delta_plain(c, proj, z, before, S0):
    """One sequence in float64: outputs, the last inputs, the last state (transposed as it is kept)."""
    n, H, G, dk, dv, C = proj.shape[0], c.H, c.G, c.dk, c.dv, c.C
    p = proj[:, 8:].to(F)
    x = torch.cat([torch.zeros(c.taps - 1, C, dtype=F) if before is None else before.to(F)[: c.taps - 1], p[:, :C]])
    y = pt.silu(pt.short_conv(x, c.conv.to(F).t()))[c.taps - 1 :]
    rep = lambda t: t.repeat_interleave(H // G, 1)
    q = rep(pt.unit_vector(y[:, : G * dk].view(n, G, dk))) * dk ** -0.5
    k = rep(pt.unit_vector(y[:, G * dk : 2 * G * dk].view(n, G, dk)))
    g = pt.channel_decays(z.to(F)[:, : H * dk], c.A.to(F), c.dt.to(F))
    o, S = pt.delta_rule(q, k, y[:, 2 * G * dk :].view(n, H, dv), torch.sigmoid(p[:, C : C + H]), g,
                         None if S0 is None else S0.to(F).transpose(1, 2))
    return o.reshape(n, H * dv), x[x.shape[0] - (c.taps - 1) :], S.transpose(1, 2)


SIZES = [(1, 1, 16, 400, 2), (4, 2, 64, 32, 4), (3, 3, 20, 12, 3), (2, 1, 128, 128, 4), (1, 1, 256, 40, 2), (5, 5, 16, 24, 1), (2, 2, 48, 72, 5),
         (4, 4, 12, 10, 4), (3, 1, 7, 9, 4), (2, 1, 132, 136, 4), (1, 1, 64, 256, 3), (1, 1, 240, 512, 2), (1, 1, 32, 520, 4)]


@pytest.mark.parametrize("decay", ["mixed", "slow", "fast", "both"])
@pytest.mark.parametrize("sizes", SIZES)
def test_delta_rule_in_chunks_portions_and_single_tokens(ops, sizes, decay):
    """A ragged batch: long portions that run as chunks side by side (from zero and from a state), short ones, first
    tokens on slots that hold garbage, single tokens behind a state; then every sequence goes on one token at a
    time. Decays from nearly one to nearly zero, also both beside one another in every key."""
    L = int(ops.ext.delta_rule_chunk())
    q_lens, starts, slots = [3 * L + 8, 9, 1, 1, L + 1, 2, 2 * L, L], [0, 5, 0, 30, 11, 0, L, 3], [3, 0, 4, 1, 2, 6, 5, 8]
    if decay != "mixed":
        q_lens, starts, slots = q_lens[:5], starts[:5], slots[:5]
    c = delta_case(*sizes, T=sum(q_lens), slots=10, decay=decay)
    b = batch(q_lens, starts, slots)
    inputs, S = c.inputs.cuda(), c.S.cuda()
    got = delta_run(ops, c, c.proj, c.z, b, inputs, S)
    at, kept = 0, []
    for n, s0, slot in zip(q_lens, starts, slots):
        ref, xs, Sn = delta_plain(c, c.proj[at : at + n], c.z[at : at + n], c.inputs[slot] if s0 else None,
                                  c.S[slot] if s0 else None)
        close(got[at : at + n], ref, 4e-6, f"sequence of {n} from {s0}")
        close(S[slot], Sn, 4e-6, "the state left behind")
        if c.taps > 1:
            close(inputs[slot], xs, 1e-7, "the inputs left behind")
        kept.append((xs, Sn))
        at += n
    assert torch.equal(S[[7, 9]].cpu(), c.S[[7, 9]]), "a slot that no sequence uses was touched"
    assert torch.equal(inputs[[7, 9]].cpu(), c.inputs[[7, 9]])
    for k in range(4):
        nb = batch([1] * len(slots), [s + n + k for s, n in zip(starts, q_lens)], slots)
        p1, z1 = rnd(len(slots), c.proj.shape[1], seed=50 + k), rnd(len(slots), c.z.shape[1], seed=80 + k)
        got = delta_run(ops, c, p1, z1, nb, inputs, S)
        for i in range(len(slots)):
            ref, xs, Sn = delta_plain(c, p1[i : i + 1], z1[i : i + 1], *kept[i])
            close(got[i : i + 1], ref, 5e-6, f"single token {k} of sequence {i}")
            kept[i] = (xs, Sn)


@pytest.mark.parametrize("cuts", [[300], [1] * 12 + [288], [2] * 20 + [260], [63, 64, 65, 66, 42], [129, 2, 1, 168], [3, 297]])
def test_delta_rule_does_not_depend_on_the_cut(ops, cuts):
    n = sum(cuts)
    c = delta_case(3, 1, 24, 40, 4, T=n, slots=2)
    inputs, S = c.inputs.cuda(), c.S.cuda()
    outs, at = [], 0
    for m in cuts:
        outs.append(delta_run(ops, c, c.proj[at : at + m], c.z[at : at + m], batch([m], [at], [1]), inputs, S))
        at += m
    ref, xs, Sn = delta_plain(c, c.proj, c.z, None, None)
    close(torch.cat(outs), ref, 4e-6)
    close(S[1], Sn, 4e-6)
    close(inputs[1], xs, 1e-7)


@pytest.mark.parametrize("gap", [1, 5, 15, 16, 17, 31, 47, 63, 64, 65, 150])
def test_a_key_is_found_again_in_the_channels_that_kept_it(ops, gap):
    """Two keys in channels of their own, written at the same time: after any distance (inside a block of the chunk,
    across blocks, across chunks) the channel without decay gives its value back exactly, the channel that
    halves at every token the right power of it, and the one that forgets at once nothing."""
    H, G, dk, dv = 1, 1, 24, 8
    n = gap + 4
    qkv = torch.zeros(n, 2 * dk + dv)
    decay = torch.ones(n, dk)
    decay[:, 1], decay[:, 2] = 0.5, 1e-30
    scal = torch.zeros(n, H, 4)
    scal[:, :, 0] = 1.0
    for t, (ch, val) in enumerate(((0, 1.0), (1, 3.0), (2, 5.0))):  # three writes, a channel each, with full steps
        qkv[t, dk + ch] = 1.0
        qkv[t, 2 * dk :] = val
        scal[t, :, 1] = 1.0
    t_read = 2 + gap
    qkv[t_read, 0], qkv[t_read, 1], qkv[t_read, 2] = 1.0, 0.25, 1.0  # one query reads all three channels
    S = rnd(1, H, dv, dk).cuda()
    out = ops.delta_rule(qkv.cuda(), scal.cuda().contiguous(), num_heads=H, num_kv_heads=G, key_dim=dk, value_dim=dv, state=S,
                         step=batch([n], [0], [0]), decay=decay.cuda()).cpu().double()
    ref = 1.0 + 0.25 * 3.0 * 0.5 ** (t_read - 1)
    assert (out[t_read] - ref).abs().max() <= 1e-6
    assert out[:2].abs().max() == 0


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W,E,top", [(7, 64, 6, 2), (40, 128, 40, 5), (4, 32, 5, 5), (30, 70, 12, 1)])
def test_router_hands_on_the_scores_as_they_are(ops, dtype, T, W, E, top):
    h, router, corr = rnd(T, W, seed=1).to(dtype), rnd(E, W, seed=2, scale=0.3), rnd(E, seed=3, scale=0.2)
    idx, wts, _ = ops.moe_route(h.cuda(), router.cuda(), E, top, False, bias=corr.cuda(), weights="softmax_of_all", normalise=False)
    z = h.to(F) @ router.to(F).T
    ri, rw = pt.choose(z, corr.to(F), top)
    assert torch.equal(idx.cpu().long(), ri)
    close(wts, rw, 1e-6)
    if top < E:
        assert not torch.equal(pt.choose(z, torch.zeros(E, dtype=F), top)[0], ri), "the correction moves a choice"


@pytest.mark.parametrize("dtype", BOTH)
@pytest.mark.parametrize("T,W,E,top,ff", [(1, 64, 4, 2, 32), (9, 96, 6, 3, 24), (40, 70, 5, 2, 18), (600, 128, 6, 2, 64)])
def test_experts_are_added_times_a_constant(ops, dtype, T, W, E, top, ff):
    from llmserve_b200.parts.base import BuildEnv
    from llmserve_b200.parts.moe import RoutedExperts, RoutedExpertsSpec

    env = BuildEnv(ops=ops, dtype=dtype, device=torch.device("cuda"), max_positions=8, branch_dtype=torch.float32)
    part = RoutedExperts(RoutedExpertsSpec(W, E, top, ff, router_weights="softmax_of_all", weight_on="output", correction=True,
                                           normalise_weights=False), env)
    params, w = {}, {}
    for k, (name, decl) in enumerate(part.param_decls().items()):
        t = rnd(*decl.shape, seed=k, scale=1.0 if "router" in name else 0.3)
        params[name] = (t.to(dtype) if decl.role == "matrix" else t).cuda().contiguous()
    for e in range(E):
        gu = params["experts.gate_up.weight"].view(E, 2 * ff, W)[e].cpu()
        w[f"e{e}.gate"], w[f"e{e}.up"] = gu[:ff], gu[ff:]
        w[f"e{e}.down"] = params["experts.down.weight"].view(E, W, ff)[e].cpu()
    w["router"], w["correction"] = params["router.weight"].cpu(), params["router.correction"].cpu()
    part.bind(params)
    h, x = rnd(T, W, seed=99).to(dtype), rnd(T, W, seed=98)
    xd = x.cuda()
    assert part.forward_into(h.cuda(), None, xd, -0.6) == []
    ref = x.to(F) - 0.6 * pt.moe(h.to(F), w, "", {"router": {"experts": E, "top": top}})
    close(xd, ref, 1e-5 if dtype == torch.float32 else 1e-2)
    ops.check_kernel_errors()


# ----------------------------------------------------------------------------- the model
def gpu_runner(folder, name, num_pages, dtype, max_num_seqs=4, max_len=512):
    from llmserve_b200.engine.runner import ModelRunner, load_model
    from llmserve_b200.ops import get_ops

    _, _, model = load_model(folder, dtype, "cuda", get_ops("cuda"), max_len)
    return ModelRunner(model, page_tokens=TANUPEL_TINY[name]["page_tokens"], num_pages=num_pages,
                       max_model_len=max_len, max_num_seqs=max_num_seqs, max_num_batched_tokens=max_len)


LENGTHS = {"T1": [5, 70, 1, 33, 49, 190, 2], "T2": [2, 40, 9, 64, 17, 100], "T3": [3, 150, 18, 77, 230]}
TOL = {"float32": (3e-4, 2e-5), "bfloat16": (0.0, 0.03)}  # (absolute, relative to the largest logit)


@pytest.fixture(scope="module")
def expected(tanupel_dirs):
    out = {}
    for name in NAMES:
        reqs = traces.make_requests(LENGTHS[name], TANUPEL_TINY[name]["config"]["vocab"], seed=5)
        out[name] = (reqs, {r: pt.model_logits(tanupel_dirs[name], t) for r, t in reqs.items()})
    return out


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
@pytest.mark.parametrize("mode", ["whole", "decode_tail", "portions", "mixed"])
def test_every_way_of_cutting_matches_plain(tanupel_dirs, expected, name, mode, dtype):
    reqs, exp = expected[name]
    runner = gpu_runner(tanupel_dirs[name], name, traces.tokens_needed(reqs) // TANUPEL_TINY[name]["page_tokens"], dtype)
    got = traces.replay(runner, getattr(traces, mode)(reqs))
    atol, rtol = TOL[dtype]
    traces.compare(got, exp, atol=atol, rtol=rtol)
    assert runner.manager.usage() == 0.0
    runner.check_kernels()


@pytest.mark.parametrize("name", NAMES)
def test_runs_of_layers_one_by_one_in_float32(tanupel_dirs, name):
    folder = tanupel_dirs[name]
    tokens = traces.make_requests([150], TANUPEL_TINY[name]["config"]["vocab"], seed=2)["r0"]
    cfg, w = pt.load(folder)
    _, after = pt.forward(tokens, w, cfg, return_layers=True)
    runner = gpu_runner(folder, name, 20, "float32")
    seen = []
    for block in runner.model.blocks:
        inner = block.forward

        def spy(x, pending, step, cache, inner=inner):
            x, pending = inner(x, pending, step, cache)
            assert pending.resolve() is None  # what the layer left for the next norm: added now
            seen.append(x.clone())
            return x, None

        block.forward = spy
    from llmserve_b200.engine.batch import StepEntry

    runner.run([StepEntry("a", tokens, [0])])
    assert len(seen) == len(pt.run_order(cfg)) == after.shape[0]
    for i, x in enumerate(seen):
        close(x, after[i], 2e-5, f"after run {i}")


def test_float32_logits_do_not_depend_on_the_cut(tanupel_dirs, expected):
    reqs, _ = expected["T1"]
    pool = traces.tokens_needed(reqs) // 16
    a = traces.replay(gpu_runner(tanupel_dirs["T1"], "T1", pool, "float32"), traces.whole(reqs))
    b = traces.replay(gpu_runner(tanupel_dirs["T1"], "T1", pool, "float32"), traces.mixed(reqs, seed=4))
    scale = max(v.abs().max().item() for v in a.values())
    assert max((a[k] - b[k]).abs().max().item() for k in a) <= 2e-5 * scale


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_from_the_first_token(tanupel_dirs, dtype):
    reqs = traces.make_requests([300], 131, seed=21)
    exp = {r: pt.model_logits(tanupel_dirs["T2"], t) for r, t in reqs.items()}
    runner = gpu_runner(tanupel_dirs["T2"], "T2", 38, dtype)
    got = traces.replay(runner, traces.decode_tail(reqs, tail=300))
    atol, rtol = TOL[dtype]
    traces.compare(got, exp, atol=atol, rtol=rtol)


def test_slots_and_pages_used_again(tanupel_dirs):
    """One state slot and just enough pages: every request runs on what the one before it left."""
    reqs = traces.make_requests([40, 37, 64, 3, 150], 167, seed=8)
    exp = {r: pt.model_logits(tanupel_dirs["T1"], t) for r, t in reqs.items()}
    runner = gpu_runner(tanupel_dirs["T1"], "T1", 10, "float32", max_num_seqs=1)
    traces.compare(traces.replay(runner, traces.portions(reqs)), exp, atol=3e-4, rtol=2e-5)


@pytest.mark.parametrize("name", NAMES)
def test_steps_that_want_some_rows_or_none(tanupel_dirs, name):
    wanted_subsets(lambda: gpu_runner(tanupel_dirs[name], name, 16, "float32"), tanupel_dirs[name],
                   TANUPEL_TINY[name]["config"]["vocab"], 3e-4)
    wanted_subsets(lambda: gpu_runner(tanupel_dirs[name], name, 16, "bfloat16"), tanupel_dirs[name],
                   TANUPEL_TINY[name]["config"]["vocab"], 0.0, 0.06)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("at", [0, 31, 32, 200, 398])
def test_a_changed_token_far_back_changes_the_last_logits_alike(tanupel_dirs, dtype, at):
    """Another token at the sequence's start, at a page's last and next first place, far back and just before: the
    engine's last logits, of a portion and single tokens behind it, follow the plain model's."""
    from llmserve_b200.engine.batch import StepEntry

    tokens = traces.make_requests([400], 300, seed=31)["r0"]
    other = list(tokens)
    other[at] = (other[at] + 17) % 300
    cfg, w = pt.load(tanupel_dirs["T3"])
    refs = [pt.forward(t, w, cfg)[-1] for t in (tokens, other)]
    runner = gpu_runner(tanupel_dirs["T3"], "T3", 26, dtype)
    got = []
    for t in (tokens, other):
        runner.run([StepEntry("a", t[:390], [])])
        for i in range(390, 399):
            runner.run([StepEntry("a", t[i : i + 1], [])])
        got.append(runner.run([StepEntry("a", t[399:], [0])])[0].double().cpu())
        runner.finish("a")
    atol, rtol = TOL[dtype]
    bound = atol + rtol * refs[0].abs().max().item()
    for g, r in zip(got, refs):
        assert (g - r).abs().max().item() <= bound
    if dtype == "float32":
        assert (refs[0] - refs[1]).abs().max().item() > 2 * bound, "the change must show"


# ----------------------------------------------------------------------------- generation
PROMPTS = [[5, 9, 90, 31, 7], list(range(40, 57)), [3] * 33, [90, 2], list(range(90))]


def llm(folder, name, dtype, **kw):
    from llmserve_b200 import LLM

    d = dict(dtype=dtype, block_size=TANUPEL_TINY[name]["page_tokens"], num_kv_blocks=64, max_model_len=256,
             max_num_seqs=8)
    d.update(kw)
    return LLM(str(folder), **d)


def greedy(n):
    from llmserve_b200 import SamplingParams

    return SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True)


@pytest.mark.parametrize("name", ["T1", "T2"])
@pytest.mark.parametrize("kw", [dict(cuda_graphs=False), dict(cuda_graphs=True),
                                dict(cuda_graphs=True, max_num_batched_tokens=24),
                                dict(cuda_graphs=True, num_kv_blocks=14, max_num_batched_tokens=16)])
def test_greedy_float32_equals_plain_greedy(tanupel_dirs, name, kw):
    """Through the entry point: the scheduler's batches, captured steps (single tokens and padded
    steps with portions), preemption by recomputation."""
    m = llm(tanupel_dirs[name], name, "float32", **kw)
    outs = m.generate(PROMPTS, greedy(12))
    for o, p in zip(outs, PROMPTS):
        assert o.outputs[0].token_ids == pt.greedy(tanupel_dirs[name], p, 12), (kw, p)


def test_greedy_bfloat16_picks_tokens_the_plain_model_also_ranks_first(tanupel_dirs):
    outs = llm(tanupel_dirs["T1"], "T1", "bfloat16", cuda_graphs=True).generate(PROMPTS, greedy(10))
    for o, p in zip(outs, PROMPTS):
        gen = o.outputs[0].token_ids
        logits = pt.model_logits(tanupel_dirs["T1"], p + gen)[len(p) - 1 : -1]
        for t, row in zip(gen, logits):
            assert float(row.max() - row[t]) <= 0.03 * float(row.abs().max())
