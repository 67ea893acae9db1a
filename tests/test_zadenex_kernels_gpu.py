"""The kernels that came with the Zadenex design, each alone against the plain float64 statement of its mechanism
(tests/plain_zadenex.py), at sizes of their own: the scaled embedding that is kept and the pass's input rows, attention whose
scores are mixed over the heads in all its kernels, the latent attention's interleaved rotation, query latent, sink and head
gates, the matrix memory (scan, finish, single tokens), the join with a constant."""
import math

import pytest
import torch

import plain_zadenex as P
from test_falisun_kernels_gpu import _Ctx as _SeqCtx, _latent_case
from test_mumopel_kernels_gpu import _Ctx, _case

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64


@pytest.fixture(scope="module")
def ops():
    from mini_llm_b200 import ops as o
    o.library()
    return o


def rnd(*shape, seed=0, scale=1.0, dtype=torch.float32):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).to(DEV)


def _tol(dtype):
    return 2e-5 if dtype == torch.float32 else 1.2e-2


def _rel(got, want):
    return (got.double().cpu() - want).abs().max().item() / max(1.0, want.abs().max().item())


# ------------------------------------------------------------------------------------------------ embedding, pass input, join
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [8, 50, 1024])
def test_scaled_embedding_and_the_rows_of_a_pass(ops, dtype, D):
    V, T = 19, 7
    table = rnd(V, D, seed=1, dtype=dtype)
    ids = torch.tensor([0, 18, 3, 3, 7, 1, 2], dtype=torch.int32, device=DEV)
    x, keep = torch.empty(T, D, device=DEV), torch.empty(T, D, device=DEV)
    ops.embed(ids, ids, table, None, x, scale=2.75, keep=keep)
    want = table.double().cpu()[ids.long().cpu()] * 2.75
    assert _rel(x, want) < 1e-7 and torch.equal(x, keep)
    y = rnd(T, D, seed=2, scale=3.0)
    for terms in (1, 2) if dtype == torch.bfloat16 else (1,):
        wide = torch.full((T, 2 * D * terms + 8), 7.0, device=DEV, dtype=dtype)
        ops.concat_terms(y, keep, wide[:, :2 * D * terms], terms)
        w = wide.double().cpu()
        both = torch.cat([y.double().cpu(), want], 1)
        got = w[:, :2 * D] + (w[:, 2 * D:4 * D] if terms == 2 else 0.0)
        # one bfloat16 term keeps 8 bits, two keep 16
        assert _rel(got, both) < {1: 1e-7 if dtype == torch.float32 else 4e-3, 2: 2.0 ** -15}[terms]
        assert torch.all(wide[:, 2 * D * terms:] == 7.0)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-6), (torch.bfloat16, 4e-5)])
@pytest.mark.parametrize("T", [1, 5, 130])
def test_a_pass_begins_with_the_residual_the_embedding_and_its_vector(ops, dtype, tol, T):
    """The part itself: W [x; x0] + s_t.  On the bfloat16 path W is bfloat16 but x and x0 keep about 16 bits: far closer
    than a product of rounded rows could be."""
    from mini_llm_b200.engine.context import Workspace
    from mini_llm_b200.parts.passes import ConcatEmbeddingInput

    class RT:
        act_dtype = dtype
    RT.ops = ops
    D, n = 56, 3
    part = ConcatEmbeddingInput(D, n)
    W, step = rnd(D, 2 * D, seed=1, scale=0.1, dtype=dtype), rnd(n, D, seed=2)
    part.bind(dict(weight=W, step=step), RT)
    ctx = _Ctx()
    ctx.ws = Workspace(torch.device(DEV), 64)
    x0 = rnd(T, D, seed=3, scale=2.0)
    for t in range(n):
        x = rnd(T, D, seed=4 + t, scale=3.0)
        want = P.enter_pass(x.double().cpu(), x0.double().cpu(), W.double().cpu(), step[t].double().cpu())
        got = part.forward(x, x0, ctx, t)
        ops.check_device_errors()
        assert got.data_ptr() == x.data_ptr() and _rel(got, want) < tol


def test_join_with_a_constant(ops):
    from mini_llm_b200.engine.context import Workspace
    from mini_llm_b200.parts.join import NormScaleJoin

    class RT:
        act_dtype = torch.float32
    RT.ops = ops
    D, T, eps = 48, 9, 1e-3
    w, ls, y, x = rnd(D, seed=1) + 1.0, rnd(D, seed=2), rnd(T, D, seed=3), rnd(T, D, seed=4)
    ctx = _Ctx()
    ctx.ws = Workspace(torch.device(DEV), 64)
    for scaled in (False, True):
        j = NormScaleJoin(D, eps, scaled=scaled, factor=-0.3)
        j.bind(dict(weight=w, scale=ls) if scaled else dict(weight=w), RT)
        got = x.clone()
        j.forward(y, got, ctx)
        want = x.double().cpu() - 0.3 * P.rms_norm(y.double().cpu(), w.double().cpu(), eps) * (ls.double().cpu() if scaled else 1.0)
        assert _rel(got, want) < 2e-6


# ------------------------------------------------------------------------------------------------ scores mixed over the heads
def _mix(H, seed=0, sharp=False):
    """Far from symmetric, entries of both signs; ``sharp``: rows sum to one, so that a key that stands out for every raw head
    stands out for every mixed one."""
    g = torch.Generator().manual_seed(seed)
    m = torch.randn(H, H, generator=g) * (0.9 / math.sqrt(H))
    if sharp:
        m = m * 0.3
        m = m + (1.0 - m.sum(1))[:, None] * torch.eye(H)[torch.randperm(H, generator=g)]
    return m


def _want(case, mix, window=None, sink=None):
    H, G, dk, dv, dtype = case["H"], case["G"], case["dk"], case["dv"], case["dtype"]
    q = case["q"].cpu().double()
    mix = mix.double()
    out = torch.zeros(q.shape[0], H * dv, dtype=F64)
    for t, (s, p) in enumerate(zip(case["token_seq"], case["positions"])):
        K, V = (x.to(dtype).double() for x in case["dense"][s])
        lo = max(0, p - window + 1) if window else 0
        raw = torch.stack([K[lo:p + 1, h // (H // G)] @ q[t, h * dk:(h + 1) * dk] for h in range(H)]) * case["scale"]
        sc = mix @ raw
        w = P.softmax_with_sink(sc[:, None, :], sink.double())[:, 0] if sink is not None else torch.softmax(sc, -1)
        for h in range(H):
            out[t, h * dv:(h + 1) * dv] = w[h] @ V[lo:p + 1, h // (H // G)]
    return out


def _run(ops, case, impl, mix, window=None, sink=None):
    H, dv = case["H"], case["dv"]
    wide = torch.zeros(case["q"].shape[0], H * dv + 8, device=DEV, dtype=case["dtype"])
    out = wide[:, 8:]
    ops.mixed_attention(case["q"], case["k_pages"], case["v_pages"], case["bt"], case["ctx"], out, num_heads=H,
                        num_kv_heads=case["G"], scale=case["scale"], mix=mix.to(DEV), window=window,
                        sink=None if sink is None else sink.to(DEV), impl=impl)
    ops.check_device_errors()
    assert torch.all(wide[:, :8] == 0)
    return out.double().cpu()


SHAPES = [(4, 2, 16, 24, 8), (3, 3, 32, 32, 16), (6, 1, 96, 40, 4), (2, 2, 8, 1, 16), (8, 2, 20, 12, 8), (1, 1, 64, 128, 16),
          (12, 3, 48, 33, 32), (5, 5, 256, 16, 16), (20, 4, 24, 130, 8), (10, 1, 8, 256, 16)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,page", SHAPES)
def test_mixed_scores_in_a_mixed_batch(ops, dtype, H, G, dk, dv, page):
    # portions that start in the middle of a page, a whole prompt, single tokens, a portion of two
    seqs = [(150, 97), (31, 31), (200, 1), (67, 2), (1, 1), (130, 65)]
    case = _case(dtype, seqs, H, G, dk, dv, page, seed=H * 100 + dk, scale=1.7 / math.sqrt(dk))
    mix = _mix(H, seed=dk)
    for window, sink in ((None, None), (24, torch.zeros(H)), (65, torch.linspace(-2.0, 3.0, H)), (1, torch.zeros(H)), (1000, None)):
        want = _want(case, mix, window, sink)
        for impl in ("rows", "split"):
            got = _run(ops, case, impl, mix, window, sink)
            assert (got - want).abs().max() < _tol(dtype) * 2 * max(1.0, want.abs().max().item()), (impl, window)


@pytest.mark.parametrize("H,G,dk,dv,page", [(3, 3, 32, 32, 16), (4, 2, 64, 128, 16), (2, 1, 128, 16, 8), (6, 2, 96, 48, 4), (8, 2, 48, 40, 16),
                                            (12, 4, 64, 64, 16), (16, 16, 32, 64, 8), (20, 4, 16, 24, 32), (32, 2, 64, 128, 16), (1, 1, 16, 8, 16)])
def test_mixed_scores_on_tensor_cores(ops, H, G, dk, dv, page):
    seqs = [(150, 97), (31, 31), (200, 1), (67, 2), (1, 1), (130, 65), (260, 129)]
    case = _case(torch.bfloat16, seqs, H, G, dk, dv, page, seed=H * 100 + dk + 1, scale=1.7 / math.sqrt(dk))
    mix = _mix(H, seed=dk)
    n0 = ops.attention_launches.get("mixed_mma", 0)
    variants = ((None, None), (24, torch.zeros(H)), (70, torch.linspace(-2.0, 3.0, H)), (1, torch.zeros(H)), (64, None))
    for window, sink in variants:
        got, want = _run(ops, case, "mma", mix, window, sink), _want(case, mix, window, sink)
        assert (got - want).abs().max() < _tol(torch.bfloat16) * 2 * max(1.0, want.abs().max().item()), window
    assert ops.attention_launches.get("mixed_mma", 0) == n0 + len(variants)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,page", SHAPES)
def test_mixed_scores_of_single_tokens(ops, dtype, H, G, dk, dv, page):
    # contexts on both sides of the window, of a chunk of keys (64) and of a page; the first tokens of a sequence
    mix = _mix(H, seed=dv)
    for window in (100, 64, 7, None):
        w = window or 300
        seqs = [(n, 1) for n in (1, 2, max(1, w - 1), w, w + 1, w + 2, 2 * w, 63, 64, 65, 128, 129, 700)]
        case = _case(dtype, seqs, H, G, dk, dv, page, seed=H * 10 + dv + w, scale=1.7 / math.sqrt(dk))
        for sink in (None, torch.zeros(H)):
            want, got = _want(case, mix, window, sink), _run(ops, case, None, mix, window, sink)
            assert (got - want).abs().max() < _tol(dtype) * 2 * max(1.0, want.abs().max().item()), window


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("impl", ["rows", "split", "mma"])
@pytest.mark.parametrize("window", [48, 112, 65, 33])
def test_keys_just_inside_and_just_outside_the_window(ops, impl, dtype, window):
    """Sharp keys at every distance around the window's edge, at page (16), key-tile (32) and chunk (64) edges and at the first
    positions.  A query sees the sharp keys at distances 0 .. window - 1 and nothing else: a key one token too far, or one
    that is left out, moves the result by O(1)."""
    if impl == "mma" and dtype != torch.bfloat16:
        pytest.skip("the tensor-core kernel is bfloat16 only")
    c = 5 * window + 9
    mix = _mix(4, seed=2, sharp=True)
    for at in ([0], [2 * window - 1], [2 * window, 15, 16], [31, 32, 3 * window + 1], [63, 64, 127, 128]):
        at = [p for p in at if p < c]
        if impl == "split":
            cases = sorted({p + d + 1 for p in at for d in (0, 1, window - 2, window - 1, window, window + 1)} & set(range(1, c + 1)))
            cases = [(n, 1) for n in cases]
        else:
            cases = [(c, window + 11), (c, c), (c - 8, 2 * window + 3), (min(at) + window + 1, 3 if min(at) + window + 1 >= 3 else 1)]
        case = _case(dtype, cases, 4, 2, 16, 16, 16, seed=6, sharp={s: [p for p in at if p < n] for s, (n, _) in enumerate(cases)})
        got, want = _run(ops, case, impl, mix, window, torch.zeros(4)), _want(case, mix, window, torch.zeros(4))
        assert (got - want).abs().max() < _tol(dtype) * 2 * max(1.0, want.abs().max().item()), at
        if len(at) == 1:                                    # the sharp key's value rows are 2: seen in full or not at all
            for t, (s, p) in enumerate(zip(case["token_seq"], case["positions"])):
                if p == at[0] + window - 1:
                    assert (got[t] - 2.0).abs().max() < 0.1
                if p == at[0] + window:
                    assert (got[t] - 2.0).abs().max() > 0.5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("impl", ["rows", "split", "mma"])
def test_a_head_takes_the_scores_that_its_row_names(ops, impl, dtype):
    """Mixing by a cyclic permutation: head h attends with the scores of head h + 1 (not h - 1: the transpose), but with its own
    values.  Raw head g has one sharp key of its own, so every head's result names the row it read."""
    if impl == "mma" and dtype != torch.bfloat16:
        pytest.skip("the tensor-core kernel is bfloat16 only")
    H, n = 4, 210
    ql = 1 if impl == "split" else 70
    case = _case(dtype, [(n, ql)], H, 2, 16, 16, 16, seed=3)
    K, V = case["dense"][0]
    q = torch.zeros(ql, H, 16)
    K *= 0.1
    sharp = [5, 77, 100, 130]                               # head g's key: direction g within its key/value head
    for g in range(H):
        q[:, g, g] = 8.0
        K[sharp[g], g // 2] = 0.0
        K[sharp[g], g // 2, g] = 30.0
    V[:] = torch.arange(n, dtype=torch.float32)[:, None, None] / 64.0
    V[:, 1] += 100.0
    case["q"] = q.reshape(ql, H * 16).to(dtype).to(DEV)
    for p in range(n):
        case["k_pages"][case["tables"][0][p // 16], :, p % 16] = K[p].to(dtype).to(DEV)
        case["v_pages"][case["tables"][0][p // 16], :, p % 16] = V[p].to(dtype).to(DEV)
    mix = torch.eye(H)[[1, 2, 3, 0]]
    got = _run(ops, case, impl, mix)
    assert (got - _want(case, mix)).abs().max() < (1e-3 if dtype == torch.float32 else 0.5)
    last = got[-1].view(H, 16)
    for h in range(H):
        row = V[sharp[(h + 1) % H], h // 2, 0].to(dtype).item()
        assert (last[h] - row).abs().max() < (1e-3 if dtype == torch.float32 else 0.5), h


def test_mixed_scores_do_not_depend_on_the_batch(ops):
    """The same token as part of a portion cut elsewhere and beside other requests: the same bits from the kernel for portions;
    alone through the single-token kernel: rounding."""
    mix = _mix(6, seed=1)
    for dtype in (torch.float32, torch.bfloat16):
        a = _case(dtype, [(200, 90)], 6, 2, 32, 32, 16, seed=5)
        impl = "mma" if dtype == torch.bfloat16 else "rows"
        full = _run(ops, a, impl, mix, 77, torch.zeros(6))
        from mini_llm_b200.engine.context import attention_tiles
        for n in (1, 2, 33):
            ctx = _Ctx()
            ctx.token_seq, ctx.positions = a["ctx"].token_seq[-n:].contiguous(), a["ctx"].positions[-n:].contiguous()
            ctx.ws, ctx.max_ctx_len, ctx.decode_only = a["ctx"].ws, 200, n == 1
            tiles = attention_tiles([n], [200 - n])
            ctx.attn_tiles, ctx.n_tiles = torch.tensor(tiles, dtype=torch.int32, device=DEV), len(tiles) // 3
            part = dict(a, q=a["q"][-n:].contiguous(), ctx=ctx)
            got = _run(ops, part, impl, mix, 77, torch.zeros(6))
            assert torch.equal(got, full[-n:]) or (got - full[-n:]).abs().max() < _tol(dtype) * 0.5
            if n == 1:
                assert (_run(ops, part, "split", mix, 77, torch.zeros(6)) - full[-1:]).abs().max() < _tol(dtype) * 2


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dn,dr,R,Q,base", [(3, 16, 8, 40, 24, 50.0), (2, 8, 16, 136, 33, 1e4), (1, 4, 4, 12, 200, 7.0), (5, 32, 64, 64, 48, 5e5)])
def test_query_latent_and_interleaved_rotation(ops, dtype, H, dn, dr, R, Q, base):
    from mini_llm_b200.parts.rotary import rotary_table
    eps, page = 1e-5, 8
    ctx = _SeqCtx([(700, 5), (3, 3), (4100, 2)])
    T, dk, row = ctx.T, R + dr, -(-(R + dr) // 8) * 8
    proj = rnd(T, Q + dk + 3, seed=5, scale=1.5, dtype=dtype)
    nw, qw = rnd(R, seed=6) * 0.3 + 1.0, rnd(Q, seed=7) * 0.3 + 1.0
    pages = torch.zeros(2 * T // page + 2, 1, page, row, dtype=dtype, device=DEV)
    slots = torch.randperm(pages.shape[0] * page, generator=torch.Generator().manual_seed(1))[:T].to(torch.int32).to(DEV)
    freq = torch.tensor(rotary_table(dr, base)[0], dtype=F64).float().to(DEV)
    cq = torch.zeros(T, Q + 5, dtype=dtype, device=DEV)
    kw = dict(dim=dn, rot_dim=dr, rank=R, rot_dims=dr, interleaved=True)
    ops.latent_prepare(proj, 0, Q, ctx, slots, freq, 1.0, nw, eps, pages, None, heads=0, write=True, dq_norm=qw, cq=cq[:, :Q], **kw)
    pos = ctx.positions.cpu().long()
    x = proj.double().cpu()
    rows = pages.view(-1, row)[slots.long()].double().cpu()
    assert _rel(cq[:, :Q], P.rms_norm(x[:, :Q], qw.double().cpu(), eps)) < _tol(dtype) and torch.all(cq[:, Q:] == 0)
    assert _rel(rows[:, :R], P.rms_norm(x[:, Q:Q + R], nw.double().cpu(), eps)) < _tol(dtype)
    assert _rel(rows[:, R:dk], P.rotate_pairs(x[:, Q + R:Q + dk], pos, dr, base)) < _tol(dtype) and torch.all(rows[:, dk:] == 0)
    q = rnd(T, H * (dn + dr) + 4, seed=8, dtype=dtype)
    qa = torch.zeros(T, H * dk, device=DEV)
    before = pages.clone()
    ops.latent_prepare(q, 0, None, ctx, slots, freq, 1.0, None, eps, None, qa, heads=H, write=False, **kw)
    qr = P.rotate_pairs(q.double().cpu()[:, :H * (dn + dr)].view(T, H, dn + dr)[..., dn:].transpose(0, 1), pos, dr, base).transpose(0, 1)
    assert _rel(qa.view(T, H, dk)[..., R:], qr) < 2e-6 and torch.equal(before, pages)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,H,N,K", [(1, 3, 40, 16), (9, 5, 1, 8), (37, 2, 136, 24), (70, 5, 8, 64), (5, 1, 65, 33), (130, 4, 64, 40)])
def test_one_gate_per_head(ops, dtype, T, H, N, K):
    y, W = rnd(T, H * K, seed=3), rnd(H, N, K, seed=2, scale=K ** -0.5, dtype=dtype)
    g = rnd(T, H + 8, seed=4, scale=2.0, dtype=dtype)
    out = torch.zeros(T, H * N, dtype=dtype, device=DEV)
    ops.headwise_linear(y, K, W, out, N, gate=g[:, 8:])
    want = torch.einsum("thk,hnk->thn", y.double().cpu().view(T, H, K), W.double().cpu()) * torch.sigmoid(g.double().cpu()[:, 8:])[..., None]
    assert _rel(out.view(T, H, N), want) < _tol(dtype)


def _sink_want(ctx, qa, dense, seqs, H, R, scale, sink):
    out, t, dk = [], 0, qa.shape[1] // H
    for s, (c, ql) in enumerate(seqs):
        rows = dense[s].double()
        for i in range(ql):
            q = qa[t].double().cpu().view(H, dk)
            w = P.softmax_with_sink(((q @ rows[:c - ql + i + 1].t()) * scale)[:, None, :], sink)[:, 0]
            out.append((w @ rows[:c - ql + i + 1, :R]).reshape(-1))
            t += 1
    return torch.stack(out)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,R,dr,page", [(3, 40, 8, 8), (10, 136, 24, 16), (1, 24, 8, 64), (17, 304, 16, 4), (2, 512, 64, 16)])
def test_latent_attention_with_a_sink(ops, dtype, H, R, dr, page):
    """Sinks from far below the scores (nothing changes) to far above them (nothing is left), through the kernel of single
    tokens and short steps and the tensor-core kernel of prompt portions; the first tokens, whose sinks weigh most."""
    from mini_llm_b200.engine.context import attention_tiles
    seqs = [(300, 45), (1, 1), (257, 1), (19, 2), (600, 70), (64, 64)]
    scale = 0.3
    ctx, qa, pages, bt, dense = _latent_case(dtype, seqs, H, R, dr, page, seed=3)
    qa = qa.to(torch.bfloat16).float()                       # so that the tensor-core kernel's queries are exact
    tiles = attention_tiles([q for _, q in seqs], [c - q for c, q in seqs])
    ctx.attn_tiles, ctx.n_tiles, ctx.decode_only = torch.tensor(tiles, dtype=torch.int32, device=DEV), len(tiles) // 3, False
    sink = torch.linspace(-30.0, 12.0, H) if H > 1 else torch.tensor([2.0])
    want = _sink_want(ctx, qa, dense, seqs, H, R, scale, sink.double())
    for impl in ("split", "mma") if dtype == torch.bfloat16 else ("split",):
        out = torch.zeros(ctx.T, H * R, device=DEV)
        ops.latent_attention(qa, pages, bt, ctx, out, heads=H, rank=R, scale=scale, sink=sink.to(DEV), impl=impl)
        assert _rel(out, want) < (2e-5 if impl == "split" else 2e-4), impl
    # single tokens: short splits, the sink counted once and not once per split
    singles = [(n, 1) for n in (1, 2, 127, 128, 129, 500)]
    ctx, qa, pages, bt, dense = _latent_case(dtype, singles, H, R, dr, page, seed=4)
    ctx.decode_only = True
    out = torch.zeros(ctx.T, H * R, device=DEV)
    ops.latent_attention(qa, pages, bt, ctx, out, heads=H, rank=R, scale=scale, sink=sink.to(DEV))
    assert _rel(out, _sink_want(ctx, qa, dense, singles, H, R, scale, sink.double())) < 2e-5


# ------------------------------------------------------------------------------------------------ matrix memory
def _memory_ctx(seqs, slots=None):
    ctx = _Ctx()
    cu = [0]
    for s in seqs:
        cu.append(cu[-1] + s)
    ctx.cu_q = torch.tensor(cu, dtype=torch.int32, device=DEV)
    ctx.S = len(seqs)
    ctx.state_slots = torch.tensor(slots if slots is not None else list(range(len(seqs))), dtype=torch.int32, device=DEV)
    ctx.token_seq = torch.tensor([i for i, s in enumerate(seqs) for _ in range(s)], dtype=torch.int32, device=DEV)
    return ctx


def _memory_cols(H, dk, dv, lead=4):
    c, at = {}, lead
    for name, n in (("g", H * dv), ("k", H * dk), ("i", H), ("q", H * dk), ("v", H * dv), ("f", H)):
        c[name] = at
        at += n + (-n) % 4
    return c, at


def _memory_case(T, H, dk, dv, seed):
    cols, width = _memory_cols(H, dk, dv)
    proj = rnd(T, width, seed=seed)
    g = torch.Generator().manual_seed(seed + 1)
    proj[:, cols["i"]:cols["i"] + H] = (torch.randn(T, H, generator=g) * 4.0).to(DEV)
    proj[:, cols["f"]:cols["f"] + H] = (torch.randn(T, H, generator=g) * 3.0 + 2.0).to(DEV)
    return proj, cols


def _memory_want(proj, cols, H, dk, dv, cap, eps, weight, state=None):
    x, T = proj.double().cpu(), proj.shape[0]
    col = lambda c, n: x[:, cols[c]:cols[c] + n]
    i = cap * torch.tanh(col("i", H) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh(col("f", H) / cap))
    o, st = P.memory_scan(col("q", H * dk).view(T, H, dk) * dk ** -0.5, col("k", H * dk).view(T, H, dk), col("v", H * dv).view(T, H, dv),
                          i, f, state)
    y = P.rms_unit(o, eps).reshape(T, H * dv) * weight.double().cpu() * torch.sigmoid(col("g", H * dv))
    return y, st


def _memory_run(ops, proj, cols, state, ctx, H, dk, dv, cap, eps, weight, step=False, dtype=torch.float32, want_cols=0):
    T = proj.shape[0]
    out = torch.zeros(T, H * dv, device=DEV, dtype=dtype)
    kw = dict(heads=H, dim=dk, vdim=dv)
    norms = dict(q_scale=dk ** -0.5, denom_eps=1e-6, eps=eps)
    if step:
        ops.mlstm_step(proj, cols, weight, state, ctx, out, cap=cap, **norms, **kw)
    else:
        raw, aux = torch.empty(T, H * dv, device=DEV), torch.empty(T, 2 * H, device=DEV)
        ops.mlstm_scan(proj, cols, state, ctx, raw, aux, cap=cap, want_cols=want_cols, **kw)
        ops.mlstm_finish(raw, aux, proj, cols, weight, state, ctx, out, **norms, **kw)
    ops.check_device_errors()
    return out


def _state_of(row, H, dk, dv):
    r = row.double().cpu()
    a, b = H * dk * dv, H * dk
    return r[:a].view(H, dk, dv), r[a:a + b].view(H, dk), r[a + b:a + b + H]


MEM = [(3, 16, 24, 5.0), (2, 64, 64, 15.0), (1, 40, 8, 8.0), (5, 8, 33, 2.0), (1, 1, 1, 4.0), (2, 96, 20, 30.0), (1, 130, 160, 6.0), (2, 12, 16, 9.0),
       (1, 256, 64, 10.0), (3, 5, 7, 3.0)]


@pytest.mark.parametrize("H,dk,dv,cap", MEM)
def test_memory_in_unequal_portions_and_batches(ops, H, dk, dv, cap):
    """Three requests whose tokens come in unequal portions over four steps, with slots used out of order and one request
    sitting a step out: outputs against the statement, the state (S, n and the running maximum) the same bits as when every
    request runs in one piece, with either number of columns per CTA, and a slot nobody owns left alone."""
    lens, plan, slots, eps = [45, 7, 33], [[17, 2, 1], [1, 0, 16], [16, 1, 15], [11, 4, 1]], [2, 0, 3], 1e-5
    proj, cols = _memory_case(sum(lens), H, dk, dv, seed=H * 7 + dk)
    weight = rnd(H * dv, seed=5) * 0.3 + 1.0
    n = H * (dk * (dv + 1) + 1)
    state = torch.zeros(4, n + 3, device=DEV)               # a wider row than needed
    state[1] = 9.0
    starts, at, got = [0, lens[0], lens[0] + lens[1]], [0, 0, 0], [[] for _ in lens]
    for k, step in enumerate(plan):
        live = [i for i, c in enumerate(step) if c]
        rows = torch.cat([torch.arange(starts[i] + at[i], starts[i] + at[i] + step[i]) for i in live]).to(DEV)
        ctx = _memory_ctx([step[i] for i in live], [slots[i] for i in live])
        out = _memory_run(ops, proj[rows], cols, state, ctx, H, dk, dv, cap, eps, weight, want_cols=(0, 32, 16, 0)[k])
        o = 0
        for i in live:
            got[i].append(out[o:o + step[i]].double().cpu())
            o += step[i]
            at[i] += step[i]
    for i, L in enumerate(lens):
        sl = slice(starts[i], starts[i] + L)
        want, st = _memory_want(proj[sl], cols, H, dk, dv, cap, eps, weight)
        assert (torch.cat(got[i]) - want).abs().max() < 5e-5 * max(1.0, want.abs().max().item()), i
        for name, a, b in zip("Snm", _state_of(state[slots[i]], H, dk, dv), st):
            assert (a - b).abs().max() < 2e-5 * max(1.0, b.abs().max().item()), (i, name)
        for wc in (16, 32):
            one = torch.zeros(4, n + 3, device=DEV)
            out = _memory_run(ops, proj[sl].contiguous(), cols, one, _memory_ctx([L], [slots[i]]), H, dk, dv, cap, eps, weight, want_cols=wc)
            assert torch.equal(one[slots[i]], state[slots[i]]), wc          # the same bits however the tokens were cut
            assert torch.equal(out.double().cpu(), torch.cat(got[i])), wc
    assert torch.all(state[1] == 9.0) and torch.all(state[:, n:][[0, 2, 3]] == 0.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv,cap", [c for c in MEM if c[1] * c[2] <= 16 * 1024])
def test_single_tokens_in_one_launch_leave_the_same_state(ops, dtype, H, dk, dv, cap):
    if not ops.mlstm_step_ok(dk, dv):
        assert dk * (-(-dv // 32) * 32) > 16 * 1024
        return
    lens, steps, eps, slots = [9, 1, 20, 3, 16], 14, 1e-5, [4, 0, 2, 1, 3]
    weight = rnd(H * dv, seed=10) * 0.3 + 1.0
    state_a = torch.zeros(5, H * (dk * (dv + 1) + 1), device=DEV)
    proj, cols = _memory_case(sum(lens), H, dk, dv, seed=dk)
    _memory_run(ops, proj, cols, state_a, _memory_ctx(lens, slots), H, dk, dv, cap, eps, weight)
    state_b = state_a.clone()
    for s in range(steps):
        p1, _ = _memory_case(5, H, dk, dv, seed=100 + s)
        ctx = _memory_ctx([1] * 5, slots)
        want = _memory_run(ops, p1, cols, state_a, ctx, H, dk, dv, cap, eps, weight)
        got = _memory_run(ops, p1, cols, state_b, ctx, H, dk, dv, cap, eps, weight, step=True, dtype=dtype)
        assert (got.double() - want.double()).abs().max() < (3e-5 if dtype == torch.float32 else 1e-2) * max(1.0, want.abs().max().item()), s
        assert torch.equal(state_a, state_b), s


def test_memory_over_long_sequences_and_extreme_gates(ops):
    """1,500 tokens with forget gates that keep nearly everything, input gates that climb to the cap and fall far below zero:
    the running maximum holds every exponential in range; heads that forget at once, that never take anything in, and whose
    maximum stays at zero."""
    H, dk, dv, cap, eps, T = 4, 32, 16, 40.0, 1e-5, 1500
    proj, cols = _memory_case(T, H, dk, dv, seed=1)
    t = torch.arange(T, dtype=torch.float32, device=DEV)
    i0, f0 = cols["i"], cols["f"]
    proj[:, i0] = 60.0 * torch.sin(t / 200.0)               # head 0: up to the cap and down again, forgetting slowly
    proj[:, f0] = 9.0
    proj[:, i0 + 1], proj[:, f0 + 1] = 3.0, -80.0           # head 1: forgets at once: the current token only
    proj[:, i0 + 2], proj[:, f0 + 2] = -100.0, 12.0         # head 2: takes next to nothing in; the maximum stays near zero
    proj[:, i0 + 3], proj[:, f0 + 3] = 0.0, 100.0           # head 3: keeps everything
    weight = rnd(H * dv, seed=3)
    state = torch.zeros(1, H * (dk * (dv + 1) + 1), device=DEV)
    out = _memory_run(ops, proj, cols, state, _memory_ctx([T]), H, dk, dv, cap, eps, weight)
    want, st = _memory_want(proj, cols, H, dk, dv, cap, eps, weight)
    assert torch.isfinite(out).all()
    # sums of 1,500 terms in 32-bit; where n . q nearly cancels the quotient magnifies them
    err = (out.double().cpu() - want).abs().max(1).values / want.abs().max()
    assert float(err.max()) < 2e-3 and float(err.median()) < 2e-5
    S, n, m = _state_of(state[0], H, dk, dv)
    # m near 36 takes a thousand steps of -1e-4 in 32-bit, each rounded to 4e-6
    assert (m - st[2]).abs().max() < 4e-3 and (m - st[2]).abs()[1:].max() < 1e-6 and abs(float(m[2])) < 0.1
    k_last, v_last = (proj[-1, cols[c] + 1 * w:cols[c] + 2 * w].double().cpu() for c, w in (("k", dk), ("v", dv)))
    assert (S[1] - k_last[:, None] * v_last).abs().max() < 1e-4
