"""The kernels that came with the Zanelorn design, each alone against the plain float64 statement of its mechanism
(tests/plain_zanelorn.py), at sizes of their own: the residual's copy for branches that read it, the norm per head before the
rotation, attention with kept first tokens and an output gate in all its kernels, retention (rotation, scan, finish, single
tokens), the selective scan (prompt portions, single tokens), the router's correction, identity experts and the shared
expert's gate, the token's own input."""
import math

import pytest
import torch

import plain_zanelorn as P
from test_falisun_kernels_gpu import _Ctx as _SeqCtx
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


def _portions(lens, slots=None, starts=None):
    """What the recurrent kernels read of a step: new tokens per request, state rows, first positions."""
    starts = [0] * len(lens) if starts is None else starts
    ctx = _SeqCtx([(a + n, n) for a, n in zip(starts, lens)], slots)
    ctx.decode_only = all(n == 1 for n in lens)
    return ctx


# ------------------------------------------------------------------------------------------------ the residual's copies
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("D", [8, 50, 1024])
def test_embedded_rows_with_a_copy_in_the_activation_dtype(ops, dtype, D):
    table = rnd(19, D, seed=1, dtype=dtype)
    ids = torch.tensor([0, 18, 3, 3, 7], dtype=torch.int32, device=DEV)
    x, h = torch.empty(5, D, device=DEV), torch.empty(5, D, device=DEV, dtype=dtype)
    ops.embed(ids, ids, table, None, x, scale=-2.75, act=h)
    want = table.double().cpu()[ids.long().cpu()] * -2.75
    assert _rel(x, want) < 1e-7 and torch.equal(h, x.to(dtype))


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,D,top", [(1, 50, 3), (9, 48, 2), (3, 2048, 5)])
def test_join_that_hands_the_new_residual_on(ops, dtype, T, D, top):
    from mini_llm_b200.engine.context import Workspace
    from mini_llm_b200.parts.join import NormScaleJoin

    class RT:
        act_dtype = dtype
    RT.ops = ops
    j = NormScaleJoin(D, 1e-3, scaled=False, factor=-0.3)
    w = rnd(D, seed=1) + 1.0
    j.bind(dict(weight=w), RT)
    ctx = _Ctx()
    ctx.ws = Workspace(torch.device(DEV), 64)
    y, x0, pairs, pw = rnd(T, D, seed=3), rnd(T, D, seed=4), rnd(T * top, D, seed=5), rnd(T, top, seed=6)
    mixed = torch.einsum("tk,tkd->td", pw.double().cpu(), pairs.double().cpu().view(T, top, D))
    for kw, v in ((dict(y=y), y.double().cpu()), (dict(y=y, pairs=(pairs, pw, top)), y.double().cpu() + mixed), (dict(y=None, pairs=(pairs, pw, top)), mixed)):
        x = x0.clone()
        h = j.forward(kw["y"], x, ctx, pairs=kw.get("pairs"), then_copy=True)
        assert _rel(x, x0.double().cpu() - 0.3 * P.rms_norm(v, w.double().cpu(), 1e-3)) < 3e-6
        assert torch.equal(h, x.to(dtype)) and (h.data_ptr() == x.data_ptr()) == (dtype == torch.float32)


# ------------------------------------------------------------------------------------------------ norm per head, rotation
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,rot,base,factor", [(6, 2, 20, 12, 8, 100.0, 3.0), (2, 2, 16, 16, 16, 20.0, 1.0), (4, 1, 8, 24, 0, 10.0, 2.0),
                                                       (1, 1, 64, 16, 64, 1e3, 8.0), (8, 2, 128, 128, 64, 1e4, 2.5), (5, 5, 6, 2, 2, 3.0, 4.0)])
def test_norm_per_head_before_the_rotation(ops, dtype, H, G, dk, dv, rot, base, factor):
    """Heads of very different sizes: one norm over the whole projection, or one after the rotation, would show."""
    from mini_llm_b200.parts.rotary import rotary_table
    T, page, eps = 23, 4, 1e-4
    nq, nk, nv = H * dk, G * dk, G * dv
    proj = rnd(T, nq + nk + nv + 3, seed=H + dk, scale=1.5).float()
    proj[:, :nq] *= torch.logspace(-2, 1, H, device=DEV).repeat_interleave(dk)
    proj[:, nq:nq + nk] *= torch.logspace(1, -1, G, device=DEV).repeat_interleave(dk)
    proj = proj.to(dtype)
    qw, kw = rnd(dk, seed=2) + 1.5, rnd(dk, seed=3) - 1.5
    g = torch.Generator().manual_seed(7)
    positions = torch.randint(0, 9000, (T,), generator=g)
    slots = torch.randperm(9 * page, generator=g)[:T].to(torch.int32)
    dkp = -(-dk // 8) * 8
    k_pages, v_pages = torch.zeros(9, G, page, dkp, device=DEV, dtype=dtype), torch.zeros(9, G, page, dv, device=DEV, dtype=dtype)
    ctx = _Ctx()
    ctx.positions = positions.to(torch.int32).to(DEV)
    freq = torch.tensor(rotary_table(rot, base, {"factor": factor})[0], dtype=F64).float().to(DEV) if rot else None
    q_out = torch.empty(T, nq, device=DEV, dtype=dtype)
    ops.qk_norm_rope(proj, 0, nq, nq + nk, ctx, q_out, k_pages, v_pages, slots.to(DEV), heads=H, kv_heads=G, head_dim=dk, v_head_dim=dv,
                     q_norm=qw, k_norm=kw, eps=eps, freq=freq, rot_dims=rot, interleaved=False, head_norm="weighted")
    ops.check_device_errors()
    x = proj.double().cpu()

    def want(lo, n, w):
        h = P.rms_norm(x[:, lo:lo + n * dk].view(T, n, dk), w.double().cpu(), eps).transpose(0, 1)
        return P.rotate_halves(h, positions, rot, base, factor).transpose(0, 1)
    wq, wk = want(0, H, qw), want(nq, G, kw)
    assert _rel(q_out.view(T, H, dk), wq) < _tol(dtype)
    for t in range(T):
        s = int(slots[t])
        assert _rel(k_pages[s // page, :, s % page, :dk], wk[t]) < _tol(dtype) and torch.all(k_pages[s // page, :, s % page, dk:] == 0)
        assert torch.equal(v_pages[s // page, :, s % page].reshape(-1), proj[t, nq + nk:nq + nk + nv])


# ------------------------------------------------------------------------------------------------ kept first tokens, gate
def _want(case, window, keep, gate=None, out_scale=1.0):
    H, G, dk, dv, dtype = case["H"], case["G"], case["dk"], case["dv"], case["dtype"]
    q = case["q"].cpu().double()
    out = torch.zeros(q.shape[0], H * dv, dtype=F64)
    for t, (s, p) in enumerate(zip(case["token_seq"], case["positions"])):
        K, V = (x.to(dtype).double() for x in case["dense"][s])
        m = P.visible(p + 1, window, keep)[p]
        o = P.softmax_attention(q[t].view(H, 1, dk), K[:p + 1].transpose(0, 1), V[:p + 1].transpose(0, 1), case["scale"], m[None])
        out[t] = o.reshape(-1)
    if gate is not None:
        out *= torch.sigmoid(gate.double().cpu())
    return out * out_scale


def _run(ops, case, impl, window, keep, gate=None, out_scale=1.0):
    H, dv = case["H"], case["dv"]
    wide = torch.zeros(case["q"].shape[0], H * dv + 8, device=DEV, dtype=case["dtype"])
    out = wide[:, 8:]
    ops.biased_attention(case["q"], case["k_pages"], case["v_pages"], case["bt"], case["ctx"], out, num_heads=H, num_kv_heads=case["G"],
                         scale=case["scale"], window=window, keep_first=keep, gate=gate, out_scale=out_scale, impl=impl)
    ops.check_device_errors()
    assert torch.all(wide[:, :8] == 0)
    return out.double().cpu()


SHAPES = [(4, 2, 16, 24, 8), (3, 3, 32, 32, 16), (6, 1, 96, 40, 4), (2, 2, 8, 1, 16), (8, 2, 24, 12, 8), (1, 1, 64, 128, 16), (5, 5, 256, 16, 16)]


def _gate(case, seed=5):
    """A column slice of a wider buffer, entries from nearly closed to open."""
    T, n = case["q"].shape[0], case["H"] * case["dv"]
    return rnd(T, n + 16, seed=seed, scale=2.5, dtype=case["dtype"])[:, 8:8 + n]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,page", SHAPES)
def test_kept_tokens_and_gate_in_a_mixed_batch(ops, dtype, H, G, dk, dv, page):
    # portions that start in the middle of a page, a whole prompt, single tokens, a portion of two
    seqs = [(150, 97), (31, 31), (200, 1), (67, 2), (1, 1), (130, 65)]
    case = _case(dtype, seqs, H, G, dk, dv, page, seed=H * 100 + dk, scale=1.7 / math.sqrt(dk))
    gate = _gate(case)
    impls = ["simt", "tiled"] + (["mma"] if dtype == torch.bfloat16 and dk % 16 == 0 and dv % 16 == 0 and dk <= 128 else [])
    for window, keep in ((24, 5), (65, 70), (1, 1), (33, 0), (64, 32), (1000, 3), (None, 0)):
        want = _want(case, window, keep, gate, 0.7)
        for impl in impls:
            got = _run(ops, case, impl, window, keep, gate, 0.7)
            assert (got - want).abs().max() < _tol(dtype) * 2 * max(1.0, want.abs().max().item()), (impl, window, keep)
    plain = _run(ops, case, "tiled", 24, 5)
    assert (plain - _want(case, 24, 5)).abs().max() < _tol(dtype) * 2 * max(1.0, plain.abs().max().item())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,page", SHAPES)
def test_kept_tokens_and_gate_of_single_tokens(ops, dtype, H, G, dk, dv, page):
    # contexts on both sides of the window, of the kept tokens, of a split (256), a tile and a page; the first tokens
    for window, keep in ((100, 7), (64, 33), (7, 300), (300, 1), (5, 256), (None, 0)):
        w = window or 300
        seqs = [(n, 1) for n in (1, 2, max(1, w - 1), w, w + 1, w + keep, w + keep + 1, 2 * w, 63, 64, 65, 256, 257, 700)]
        case = _case(dtype, seqs, H, G, dk, dv, page, seed=H * 10 + dv + w, scale=1.7 / math.sqrt(dk))
        gate = _gate(case)
        want, got = _want(case, window, keep, gate), _run(ops, case, None, window, keep, gate)
        assert (got - want).abs().max() < _tol(dtype) * 2 * max(1.0, want.abs().max().item()), (window, keep)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("impl", ["simt", "tiled", "split", "mma"])
@pytest.mark.parametrize("window,keep", [(48, 5), (65, 16), (33, 40), (112, 64), (20, 1)])
def test_keys_at_the_edges_of_the_kept_tokens_and_the_window(ops, impl, dtype, window, keep):
    """Sharp keys just inside and just outside the kept tokens and at every distance around the window's edge, at page, tile and
    split edges: a key one token too far, or one that is left out, moves the result by O(1)."""
    if impl == "mma" and dtype != torch.bfloat16:
        pytest.skip("the tensor-core kernel is bfloat16 only")
    c = 5 * window + 2 * keep + 9
    for at in ([keep - 1], [keep], [2 * window + keep], [0, 15, 16], [31, 32, 3 * window + 1], [63, 64, 127, 128, keep + 1]):
        at = sorted({p for p in at if 0 <= p < c})
        if impl == "split":
            cases = sorted({p + d + 1 for p in at for d in (0, 1, window - 2, window - 1, window, window + 1, 3 * window)} & set(range(1, c + 1)))
            cases = [(n, 1) for n in cases]
        else:
            cases = [(c, window + 11), (c, c), (c - 8, min(2 * window + 3, c - 8)), (min(at) + window + 1, min(3, min(at) + window + 1))]
        case = _case(dtype, cases, 4, 2, 16, 16, 16, seed=6, sharp={s: [p for p in at if p < n] for s, (n, _) in enumerate(cases)})
        got, want = _run(ops, case, impl, window, keep), _want(case, window, keep)
        assert (got - want).abs().max() < _tol(dtype) * 2 * max(1.0, want.abs().max().item()), at
        if len(at) == 1:                                    # the sharp key's value rows are 2: seen in full or not at all
            for t, (s, p) in enumerate(zip(case["token_seq"], case["positions"])):
                if p >= at[0] + window:
                    seen = (got[t] - 2.0).abs().max() < 0.1
                    assert bool(seen) == (at[0] < keep), (p, at)


def test_attention_with_kept_tokens_does_not_depend_on_the_batch(ops):
    from mini_llm_b200.engine.context import attention_tiles
    for dtype in (torch.float32, torch.bfloat16):
        a = _case(dtype, [(300, 190)], 6, 2, 32, 32, 16, seed=5)
        full = _run(ops, a, None, 77, 9)
        for n in (1, 2, 33, 120):
            ctx = _Ctx()
            ctx.token_seq, ctx.positions = a["ctx"].token_seq[-n:].contiguous(), a["ctx"].positions[-n:].contiguous()
            ctx.ws, ctx.max_ctx_len, ctx.decode_only = a["ctx"].ws, 300, n == 1
            tiles = attention_tiles([n], [300 - n])
            ctx.attn_tiles, ctx.n_tiles = torch.tensor(tiles, dtype=torch.int32, device=DEV), len(tiles) // 3
            part = dict(a, q=a["q"][-n:].contiguous(), ctx=ctx)
            assert (_run(ops, part, None, 77, 9) - full[-n:]).abs().max() < _tol(dtype) * 2


# ------------------------------------------------------------------------------------------------ retention
def _ret_case(T, H, dk, dv, seed):
    nk, nv = H * dk, H * dv
    cols = {"q": 0, "k": nk, "v": 2 * nk, "g": 2 * nk + nv}
    proj = rnd(T, -(-(2 * nk + 2 * nv) // 4) * 4 + 4, seed=seed)
    proj[:, nk:2 * nk] = 0.6 * proj[:, nk:2 * nk] + 0.8 * proj[:, :nk]       # keys lean towards the queries
    return proj, cols


def _ret_want(proj, cols, H, dk, dv, decay, positions, rot, base, eps, state=None):
    T = proj.shape[0]
    x = proj.double().cpu()

    def part(c, d):
        return x[:, cols[c]:cols[c] + H * d].view(T, H, d)

    def turned(c):
        return P.rotate_halves(part(c, dk).transpose(0, 1), positions, rot, base).transpose(0, 1)
    o, S = P.retention_scan(turned("q"), turned("k") * dk ** -0.5, part("v", dv), decay, state)
    return P.rms_unit(o, eps).reshape(T, H * dv) * P.silu(part("g", dv).reshape(T, H * dv)), S


def _ret_run(ops, proj, cols, decay, state, ctx, H, dk, dv, rot, base, eps, step=False, dtype=torch.float32, want_cols=0):
    from mini_llm_b200.parts.rotary import rotary_table
    freq = torch.tensor(rotary_table(rot, base)[0], dtype=F64).float().to(DEV) if rot else None
    out = torch.zeros(proj.shape[0], H * dv, device=DEV, dtype=dtype)
    r, z = dict(freq=freq, rot_dims=rot, k_scale=dk ** -0.5), dict(heads=H, dim=dk, vdim=dv)
    if step:
        before = proj.clone()
        ops.retention_step(proj, cols, decay, state, ctx, out, eps=eps, **r, **z)
        assert torch.equal(before, proj)
    else:
        p = proj.clone()
        ops.rotate_heads(p, cols["q"], cols["k"], ctx, heads=H, dim=dk, **r)
        raw = torch.empty(proj.shape[0], H * dv, device=DEV)
        ops.retention_scan(p, cols, decay, state, ctx, raw, want_cols=want_cols, **z)
        ops.retention_finish(raw, p, cols["g"], out, heads=H, vdim=dv, eps=eps)
    ops.check_device_errors()
    return out


RET = [(3, 16, 24, 16, 50.0), (2, 64, 64, 32, 1e4), (1, 40, 8, 12, 7.0), (5, 8, 33, 0, 2.0), (1, 1, 1, 0, 3.0), (2, 96, 20, 96, 1e3),
       (1, 130, 160, 2, 10.0), (1, 256, 256, 128, 1e4), (3, 5, 7, 4, 30.0), (2, 128, 256, 128, 5e5)]


def _decays(H):
    return [0.5, 0.97, 0.9995, 0.0, 1.0][:H] if H > 1 else [0.98]


@pytest.mark.parametrize("H,dk,dv,rot,base", RET)
def test_retention_in_unequal_portions_and_batches(ops, H, dk, dv, rot, base):
    """Three requests whose tokens come in unequal portions over four steps, with slots used out of order and one request
    sitting a step out: outputs against the statement, states the same bits as when every request runs in one piece, with
    either number of columns per CTA, and a slot nobody owns left alone."""
    lens, plan, slots, eps = [45, 7, 33], [[17, 2, 1], [1, 0, 16], [16, 1, 15], [11, 4, 1]], [2, 0, 3], 1e-5
    proj, cols = _ret_case(sum(lens), H, dk, dv, seed=H * 7 + dk)
    values = _decays(H)
    decay = torch.tensor(values, device=DEV)
    n = H * dk * dv
    state = torch.zeros(4, n + 3, device=DEV)               # a wider row than needed
    state[1] = 9.0
    starts, at, got = [0, lens[0], lens[0] + lens[1]], [0, 0, 0], [[] for _ in lens]
    for k, step in enumerate(plan):
        live = [i for i, c in enumerate(step) if c]
        rows = torch.cat([torch.arange(starts[i] + at[i], starts[i] + at[i] + step[i]) for i in live]).to(DEV)
        ctx = _portions([step[i] for i in live], [slots[i] for i in live], [at[i] for i in live])
        out = _ret_run(ops, proj[rows], cols, decay, state, ctx, H, dk, dv, rot, base, eps, want_cols=(0, 32, 16, 0)[k])
        o = 0
        for i in live:
            got[i].append(out[o:o + step[i]].double().cpu())
            o += step[i]
            at[i] += step[i]
    for i, L in enumerate(lens):
        sl = slice(starts[i], starts[i] + L)
        want, S = _ret_want(proj[sl], cols, H, dk, dv, [float(torch.tensor(v)) for v in values], torch.arange(L), rot, base, eps)
        assert (torch.cat(got[i]) - want).abs().max() < 1e-4 * max(1.0, want.abs().max().item()), i
        assert (state[slots[i], :n].double().cpu().view(H, dk, dv) - S).abs().max() < 2e-5 * max(1.0, S.abs().max().item()), i
        for wc in (16, 32):
            one = torch.zeros(4, n + 3, device=DEV)
            out = _ret_run(ops, proj[sl].contiguous(), cols, decay, one, _portions([L], [slots[i]]), H, dk, dv, rot, base, eps, want_cols=wc)
            assert torch.equal(one[slots[i]], state[slots[i]]), wc          # the same bits however the tokens were cut
            assert torch.equal(out.double().cpu(), torch.cat(got[i])), wc
    assert torch.all(state[1] == 9.0) and torch.all(state[:, n:][[0, 2, 3]] == 0.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv,rot,base", RET)
def test_retention_of_single_tokens_in_one_launch_leaves_the_same_state(ops, dtype, H, dk, dv, rot, base):
    if not ops.retention_step_ok(dk, dv):
        assert dk * (-(-dv // 32) * 32) > 32 * 1024
        return
    lens, steps, eps, slots = [9, 1, 20, 3, 16], 14, 1e-5, [4, 0, 2, 1, 3]
    decay = torch.tensor(_decays(H), device=DEV)
    state_a = torch.zeros(5, H * dk * dv, device=DEV)
    proj, cols = _ret_case(sum(lens), H, dk, dv, seed=dk)
    _ret_run(ops, proj, cols, decay, state_a, _portions(lens, slots), H, dk, dv, rot, base, eps)
    state_b = state_a.clone()
    for s in range(steps):
        p1, _ = _ret_case(5, H, dk, dv, seed=100 + s)
        ctx = _portions([1] * 5, slots, [n + s for n in lens])
        want = _ret_run(ops, p1, cols, decay, state_a, ctx, H, dk, dv, rot, base, eps)
        got = _ret_run(ops, p1, cols, decay, state_b, ctx, H, dk, dv, rot, base, eps, step=True, dtype=dtype)
        assert (got.double() - want.double()).abs().max() < (3e-4 if dtype == torch.float32 else 1.2e-2) * max(1.0, want.abs().max().item()), s
        # the rotation's products may round apart in the last bit where the compiler fuses them differently
        assert (state_a - state_b).abs().max() < 2e-6 * max(1.0, float(state_a.abs().max())), s


def test_retention_over_long_sequences(ops):
    """1,500 tokens: a head that keeps everything, one that forgets at once, and a key far back that only the slow heads still
    answer."""
    H, dk, dv, T, eps = 3, 32, 16, 1500, 1e-5
    values = [1.0, 0.0, 0.9990234375]
    proj, cols = _ret_case(T, H, dk, dv, seed=1)
    proj[:, cols["q"]:cols["v"]] *= 0.1
    proj[40, cols["k"]:cols["v"]] = 20.0                    # one key that stands out, met by every later query
    proj[:, cols["q"]:cols["k"]] += 1.0
    state = torch.zeros(1, H * dk * dv, device=DEV)
    decay = torch.tensor(values, device=DEV)
    out = _ret_run(ops, proj, cols, decay, state, _portions([T]), H, dk, dv, 0, 10.0, eps)
    want, S = _ret_want(proj, cols, H, dk, dv, values, torch.arange(T), 0, 10.0, eps)
    err = (out.double().cpu() - want).abs().max(1).values / want.abs().max()
    assert float(err.max()) < 1e-3 and float(err.median()) < 1e-5
    assert (state[0].double().cpu().view(H, dk, dv) - S).abs().max() < 1e-4 * S.abs().max()
    u = P.rms_unit(proj[40, cols["v"]:cols["g"]].double().cpu().view(H, dv), eps)
    r = (out[1200].double().cpu() / P.silu(proj[1200, cols["g"]:cols["g"] + H * dv].double().cpu())).view(H, dv)
    for h, far in ((0, True), (1, False), (2, True)):       # does the head still give the far key's value?
        cos = float((r[h] * u[h]).sum() / r[h].norm() / u[h].norm())
        assert (cos > 0.9) == far, (h, cos)


# ------------------------------------------------------------------------------------------------ selective scan
def _sel_case(T, C, N, R, seed, dtype):
    g = torch.Generator().manual_seed(seed)
    x, z = rnd(T, C + 5, seed=seed, dtype=dtype)[:, 2:2 + C], rnd(T, C + 3, seed=seed + 1, dtype=dtype)[:, :C]
    low = rnd(T, -(-max(R + 2 * N, R + 8) // 8) * 8, seed=seed + 2, dtype=dtype)
    W = rnd(C, R, seed=3, scale=1.0 / math.sqrt(R), dtype=dtype)
    A = -torch.exp(torch.empty(C, N).uniform_(-4.0, 1.5, generator=torch.Generator().manual_seed(4))).to(DEV)
    skip, bias = rnd(C, seed=5), rnd(C, seed=6) - 1.5
    del g
    return dict(x=x, z=z, low=low, W=W, A=A, skip=skip, bias=bias, R=R, N=N, C=C)


def _sel_want(c, rows, out_scale, state=None):
    R, N = c["R"], c["N"]
    d = {k: c[k].double().cpu() for k in ("W", "A", "skip", "bias")}
    x, z, low = (c[k][rows].double().cpu() for k in ("x", "z", "low"))
    dt = P.softplus(low[:, :R] @ d["W"].T + d["bias"])
    y, S = P.selective_scan(x, dt, d["A"], low[:, R:R + N], low[:, R + N:R + 2 * N], d["skip"], state)
    return y * P.silu(z) * out_scale, S


def _sel_run(ops, c, rows, state, ctx, out_scale, step=False):
    R, N, C = c["R"], c["N"], c["C"]
    wide = torch.zeros(len(rows), C + 7, device=DEV, dtype=c["x"].dtype)
    out = wide[:, 3:3 + C]
    x, z, low = c["x"][rows], c["z"][rows], c["low"][rows]
    args = (z, c["A"], c["skip"], c["bias"], state, ctx, out)
    if step:
        W = torch.zeros(C, -(-R // 8) * 8, device=DEV, dtype=x.dtype)
        W[:, :R] = c["W"]
        ops.selective_step(x, low, R, R, R + N, W, *args, out_scale=out_scale)
    else:
        dt = (low[:, :R].float() @ c["W"].float().T).contiguous()
        ops.selective_scan(x, dt, low, R, R + N, *args, out_scale=out_scale)
    ops.check_device_errors()
    assert torch.all(wide[:, :3] == 0) and torch.all(wide[:, 3 + C:] == 0)
    return out


SEL = [(48, 10, 5), (320, 16, 20), (1, 1, 1), (37, 3, 2), (130, 24, 12), (70, 5, 8), (40, 64, 3), (24, 100, 33), (9, 131, 16), (20, 256, 7), (96, 32, 16)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,N,R", SEL)
def test_selective_scan_in_unequal_portions_and_batches(ops, dtype, C, N, R):
    """As for retention: outputs against the statement, states and outputs the same bits as when every request runs in one piece."""
    lens, plan, slots, f = [45, 7, 34], [[17, 2, 1], [1, 0, 16], [16, 1, 16], [11, 4, 1]], [2, 0, 3], -0.7
    c = _sel_case(sum(lens), C, N, R, seed=C + N, dtype=dtype)
    n = C * N
    state = torch.zeros(4, n + 3, device=DEV)
    state[1] = 9.0
    starts, at, got = [0, lens[0], lens[0] + lens[1]], [0, 0, 0], [[] for _ in lens]
    for step in plan:
        live = [i for i, k in enumerate(step) if k]
        rows = torch.cat([torch.arange(starts[i] + at[i], starts[i] + at[i] + step[i]) for i in live]).to(DEV)
        out = _sel_run(ops, c, rows, state, _portions([step[i] for i in live], [slots[i] for i in live]), f)
        o = 0
        for i in live:
            got[i].append(out[o:o + step[i]].clone())
            o += step[i]
            at[i] += step[i]
    for i, L in enumerate(lens):
        rows = torch.arange(starts[i], starts[i] + L, device=DEV)
        want, S = _sel_want(c, rows, f)
        assert _rel(torch.cat(got[i]), want) < _tol(dtype) * 2, i
        # on the bfloat16 path the exponentials are one instruction, good to a few units of the last place of 32-bit
        assert (state[slots[i], :n].double().cpu().view(C, N) - S).abs().max() < 2e-5 * max(1.0, S.abs().max().item()), i
        one = torch.zeros(4, n + 3, device=DEV)
        out = _sel_run(ops, c, rows, one, _portions([L], [slots[i]]), f)
        if not torch.equal(one[slots[i]], state[slots[i]]):         # step sizes come from a library product here: its row count may matter
            assert (one[slots[i]] - state[slots[i]]).abs().max() < 1e-5 * max(1.0, float(one.abs().max()))
        assert (out.double() - torch.cat(got[i]).double()).abs().max() < _tol(dtype) * max(1.0, want.abs().max().item())
    assert torch.all(state[1] == 9.0) and torch.all(state[:, n:][[0, 2, 3]] == 0.0)


def test_selective_scan_bits_do_not_depend_on_the_cut(ops):
    for dtype in (torch.float32, torch.bfloat16):
        for C, N in ((48, 10), (40, 16), (12, 40), (8, 200)):
            T = 75
            c = _sel_case(T, C, N, 4, seed=1, dtype=dtype)
            dt = rnd(T, C, seed=9)
            args = dict(out_scale=1.0)
            whole, cut = torch.zeros(1, C * N, device=DEV), torch.zeros(1, C * N, device=DEV)
            a, b = torch.zeros(T, C, device=DEV, dtype=dtype), torch.zeros(T, C, device=DEV, dtype=dtype)
            ops.selective_scan(c["x"], dt, c["low"], 4, 4 + N, c["z"], c["A"], c["skip"], c["bias"], whole, _portions([T]), a, **args)
            at = 0
            for k in (3, 1, 17, 2, 16, 15, 21):
                s = slice(at, at + k)
                ops.selective_scan(c["x"][s], dt[s], c["low"][s], 4, 4 + N, c["z"][s], c["A"], c["skip"], c["bias"], cut, _portions([k], [0], [at]), b[s], **args)
                at += k
            assert at == T and torch.equal(a, b) and torch.equal(whole, cut), (dtype, C, N)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,N,R", SEL)
def test_selective_scan_of_single_tokens_in_one_launch(ops, dtype, C, N, R):
    lens, steps, slots, f = [9, 1, 20, 3], 12, [3, 0, 2, 1], 1.3
    c = _sel_case(sum(lens), C, N, R, seed=3, dtype=dtype)
    state_a = torch.zeros(4, C * N, device=DEV)
    _sel_run(ops, c, torch.arange(sum(lens), device=DEV), state_a, _portions(lens, slots), f)
    state_b = state_a.clone()
    rows = torch.arange(4, device=DEV)
    for s in range(steps):
        c1 = dict(_sel_case(4, C, N, R, seed=50 + s, dtype=dtype), A=c["A"], skip=c["skip"], bias=c["bias"], W=c["W"])
        ctx = _portions([1] * 4, slots)
        want = _sel_run(ops, c1, rows, state_a, ctx, f)
        got = _sel_run(ops, c1, rows, state_b, ctx, f, step=True)
        assert (got.double() - want.double()).abs().max() < _tol(dtype) * max(1.0, float(want.abs().max())), s
        assert (state_a - state_b).abs().max() < 1e-5 * max(1.0, float(state_a.abs().max())), s


def test_a_channel_that_keeps_and_one_that_forgets(ops):
    """2,000 tokens: a rate of nearly zero still holds the first token's share, a large one holds the current token only."""
    T, C, N = 2000, 16, 4
    for dtype in (torch.float32, torch.bfloat16):
        c = _sel_case(T, C, N, 8, seed=2, dtype=dtype)
        c["A"] = c["A"].clone()
        c["A"][0], c["A"][1] = -1e-6, -1e4
        c["x"] = c["x"] * 0.01
        c["x"][3, 0] = 50.0                                 # one input far back that stands out
        state = torch.zeros(1, C * N, device=DEV)
        out = _sel_run(ops, c, torch.arange(T, device=DEV), state, _portions([T]), 1.0)
        want, S = _sel_want(c, torch.arange(T), 1.0)
        assert _rel(out, want) < (2e-4 if dtype == torch.float32 else 1.2e-2)
        st = state.double().cpu().view(C, N)
        assert (st - S).abs().max() < 3e-4 * S.abs().max() and st[0].abs().max() > 100 * st[1].abs().max()


@pytest.mark.parametrize("taps", [1, 2, 4])
def test_convolution_with_outputs_in_the_activation_dtype(ops, taps):
    C, lens, dtype = 40, [9, 1, 2], torch.bfloat16
    proj = rnd(sum(lens), C + 8, seed=1, dtype=dtype)
    w, b = rnd(C, taps, seed=2), rnd(C, seed=3)
    state = torch.zeros(3, (taps - 1) * C + 5, device=DEV)
    out = torch.zeros(sum(lens), C, device=DEV, dtype=dtype)
    ops.ssd_conv(proj, 8, w, b, state, 5, _portions(lens), out)
    at = 0
    for n in lens:
        u = proj[at:at + n, 8:].double().cpu()
        assert _rel(out[at:at + n], P.silu(P.causal_conv(u, w.double().cpu(), b.double().cpu()))) < _tol(dtype)
        at += n
    one = torch.zeros(3, C, device=DEV, dtype=dtype)
    nxt = rnd(3, C + 8, seed=7, dtype=dtype)
    before = [torch.cat([proj[a:a + n, 8:], nxt[i:i + 1, 8:]]).double().cpu() for i, (a, n) in enumerate(zip((0, 9, 10), lens))]
    ops.ssd_conv(nxt, 8, w, b, state, 5, _portions([1, 1, 1]), one)
    for i, u in enumerate(before):
        assert _rel(one[i], P.silu(P.causal_conv(u, w.double().cpu(), b.double().cpu()))[-1]) < _tol(dtype)


# ------------------------------------------------------------------------------------------------ routing, identity experts
@pytest.mark.parametrize("T", [1, 16, 50])
@pytest.mark.parametrize("E,identity,top,D", [(7, 3, 2, 64), (12, 0, 5, 50), (1, 1, 2, 8), (40, 24, 8, 96), (300, 100, 3, 32)])
def test_router_with_a_correction_of_the_choice(ops, T, E, identity, top, D):
    """The choice follows score + correction, the weights the scores alone and undivided; the shared expert's gate beside it.
    Two equal choice scores: the lower index."""
    n = E + identity
    h, W, sg = rnd(T, D, seed=1), rnd(n, D, seed=2, scale=2.0 / math.sqrt(D)), rnd(1, D, seed=4, scale=0.3)
    corr = rnd(n, seed=3, scale=0.3)
    idx, wts, gate = torch.zeros(T, top, dtype=torch.int32, device=DEV), torch.zeros(T, top, device=DEV), torch.zeros(T, 1, device=DEV)
    off, order = torch.zeros(1, n + 1, dtype=torch.int32, device=DEV), torch.zeros(T, top, dtype=torch.int32, device=DEV)
    ops.moe_route(h, W, idx, wts, off, order, top=top, correction=corr, renorm=False, gate_weight=sg, gate=gate)
    ops.check_device_errors()
    z = h.double().cpu() @ W.double().cpu().T
    wi, ww = P.choose(z, corr.double().cpu(), top)
    plain, _ = P.choose(z, torch.zeros(n, dtype=F64), top)
    assert torch.equal(idx.cpu().long(), wi) and _rel(wts, ww) < 3e-6
    assert n == top or T < 16 or not torch.equal(plain, wi)                 # the correction changes the choice
    assert _rel(gate, torch.sigmoid(h.double().cpu() @ sg.double().cpu().T)) < 3e-6
    flat = idx.cpu().reshape(-1)
    assert torch.equal(order.cpu().reshape(-1).long(), torch.sort(flat, stable=True).indices)
    assert torch.equal(off.cpu().reshape(-1).long(), torch.tensor([int((flat < e).sum()) for e in range(n + 1)]))
    ops.moe_route(torch.zeros_like(h), W, idx, wts, off, order, top=top, correction=torch.zeros_like(corr), renorm=False)
    assert torch.equal(idx.cpu()[0], torch.arange(top, dtype=torch.int32)) and _rel(wts, torch.full((T, top), 1.0 / n, dtype=F64)) < 1e-6


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T", [3, 70])
@pytest.mark.parametrize("E,identity,top,D,F,shared", [(5, 3, 2, 64, 24, 40), (4, 0, 3, 48, 56, None), (1, 4, 5, 32, 8, 8), (6, 2, 2, 50, 13, 9), (3, 60, 4, 72, 16, None)])
def test_feed_forward_with_identity_experts_and_a_gated_shared_one(ops, dtype, T, E, identity, top, D, F, shared):
    from mini_llm_b200.engine.context import Workspace
    from mini_llm_b200.parts.moe import MoEFeedForward

    class RT:
        act_dtype = dtype
    RT.ops = ops
    part = MoEFeedForward(D, E, top, F, shared_size=shared, activation="swiglu_clamp", limit=0.9, shared_limit=1.6 if shared else None, alpha=1.702,
                          correction=True, renorm=False, identity=identity, shared_gate=shared is not None)
    g = torch.Generator().manual_seed(T + E)
    params, w = {}, {}
    for name, ps in part.param_specs().items():
        t = torch.randn(ps.shape, generator=g) * (0.1 if name == "correction" else 2.0 / math.sqrt(ps.shape[-1]))
        t = t.to(dtype).to(DEV) if ps.role == "matrix" else t.to(DEV)
        params[name] = t
        w[name.replace("expert", "e")] = t.double().cpu()
    part.bind(params, RT)
    ctx = _Ctx()
    ctx.ws = Workspace(torch.device(DEV), 64)
    h = rnd(T, D, seed=8, dtype=dtype)
    m = dict(router=dict(experts=E, top=top), expert=dict(limit=0.9), shared=dict(limit=1.6) if shared else None)
    want = P.moe(h.double().cpu(), w, m, P.to_bf16 if dtype == torch.bfloat16 else P._keep)
    y = rnd(T, D, seed=9)
    base = y.double().cpu()
    part.forward(h, ctx, y)
    ops.check_device_errors()
    assert _rel(y, base + want) < _tol(dtype)
    part.forward(h, ctx, y, accumulate=False)
    assert _rel(y, want) < _tol(dtype)
    had, (pairs, wts, k) = part.forward_pairs(h, ctx, y)
    both = torch.einsum("tk,tkd->td", wts.double().cpu(), pairs.double().cpu().view(T, k, D)) + (y.double().cpu() if had else 0.0)
    assert had == (shared is not None) and _rel(both, want) < _tol(dtype)
    idx, _ = P.choose(h.double().cpu() @ w["router"].T, w["correction"], top)
    assert identity == 0 or T < 16 or bool((idx >= E).any())                # identity experts are among the chosen
    for t in range(T):                                                      # and give exactly their input back
        for j in range(top):
            if idx[t, j] >= E:
                assert torch.equal(pairs[t * top + j], h[t].float())


# ------------------------------------------------------------------------------------------------ the token's own input
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,D,d,parts", [(1, 64, 12, 3), (16, 50, 7, 2), (9, 1024, 128, 2), (40, 96, 16, 4), (3, 40, 1, 1)])
def test_side_input_of_every_layer(ops, dtype, T, D, d, parts):
    """Every layer reads its own columns of the token's row: columns of another layer, or another token's row, would show."""
    from mini_llm_b200.engine.context import Workspace
    from mini_llm_b200.parts.side import SideTable, TokenSideBranch

    class RT:
        act_dtype = dtype
    RT.ops = ops
    V = 23
    table = SideTable(V, parts, d)
    rows = rnd(V, parts * d, seed=1, dtype=dtype) + torch.arange(parts, device=DEV).repeat_interleave(d).to(dtype)
    table.bind(dict(table=rows), RT)
    ctx = _Ctx()
    ctx.ws = Workspace(torch.device(DEV), 64)
    ids = torch.randint(0, V, (T,), generator=torch.Generator().manual_seed(T))
    ctx.token_ids = ids.to(torch.int32).to(DEV)
    h = rnd(T, D, seed=2, dtype=dtype)
    store = P.to_bf16 if dtype == torch.bfloat16 else P._keep
    for i in range(parts):
        b = TokenSideBranch(D, d, i)
        gate, proj = rnd(d, D, seed=3 + i, scale=1.0 / math.sqrt(D), dtype=dtype), rnd(D, d, seed=9 + i, scale=1.0 / math.sqrt(d), dtype=dtype)
        b.bind(dict(gate_weight=gate, proj_weight=proj), RT)
        b.attach(table)
        y = torch.full((T, D), 7.0, device=DEV)
        b.forward(h, ctx, y)
        ops.check_device_errors()
        e = rows.double().cpu()[ids][:, i * d:(i + 1) * d]
        want = store(P.gelu_tanh(h.double().cpu() @ gate.double().cpu().T) * e) @ proj.double().cpu().T
        assert _rel(y, want) < _tol(dtype)
