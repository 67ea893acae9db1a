"""Zadenex without a GPU: the configuration reader and its errors, the model description (joins, passes, cache needs, tensor
names), a state row that is used again, the random-weights folder, and the plain statement against itself."""
import copy
import json
import math

import pytest
import torch

import plain_zadenex as P
from zadenex_models import CFG_A, CFG_B, attn, config, latent, layer, make_tensors, mlstm

F64 = torch.float64


def _spec(cfg):
    import mini_llm_b200  # noqa: F401
    from mini_llm_b200.config.base import config_from_dict, get_architecture
    c = config_from_dict(cfg)
    return c, get_architecture(c.architecture).build_spec(c)


def test_every_size_is_read_per_layer():
    c, spec = _spec(CFG_A)
    assert c.architecture == "Zadenex" and (c.vocab, c.width, c.norm_eps, c.embedding_scale, c.residual_mult) == (97, 64, 1e-5, 1.5, 0.7)
    a, b, d, e = (l.mixer for l in c.layers)
    assert (a.heads, a.dim, a.vdim, a.gate_cap) == (3, 16, 24, 5.0) and (e.heads, e.dim, e.vdim, e.gate_cap) == (1, 40, 8, 15.0)
    assert (b.heads, b.kv_heads, b.dim, b.vdim, b.scale, b.window) == (8, 2, 20, 12, 0.3, 25)
    assert (d.heads, d.dim, d.rot_dim, d.vdim, d.q_rank, d.kv_rank, d.scale, d.rot_dims, d.rot_base) == (5, 12, 8, 20, 24, 40, 0.35, 8, 100.0)
    assert [l.mlp.ff if l.mlp else None for l in c.layers] == [72, 40, 56, None]
    assert [l.mixer.kind for l in spec.layers] == ["matrix_memory", "mixed_score_attention", "latent_attention", "matrix_memory"]
    assert all(l.arrangement == "sandwich" and l.mixer_join.params["factor"] == 0.7 and not l.mixer_join.params["scaled"] for l in spec.layers)
    assert spec.layers[3].ff is None and spec.layers[3].ff_join is None and r"^l3\.norm2b?$" in spec.ignored_tensors
    m = spec.layers[1].mixer.params
    assert (m["window"], m["bias"], m["out_bias"], m["sink"]) == (25, True, True, "zero")
    m = spec.layers[2].mixer.params
    assert (m["q_rank"], m["gate"], m["sink"], m["rot_interleaved"]) == (24, "head", True, True)
    m = spec.layers[0].mixer.params
    assert (m["gate_cap"], m["denom_eps"], m["norm_eps"]) == (5.0, 1e-6, 1e-5)
    f = spec.layers[0].ff.params
    assert (f["activation"], f["bias"], f["inner_size"]) == ("gelu_tanh", True, 72)
    assert spec.embedding.params["scale"] == 1.5 and spec.embedding.params["keep"] and spec.head.kind == "linear"


def test_passes_have_caches_of_their_own():
    c, spec = _spec(CFG_A)
    assert [(e.layer, e.enters_pass, e.private_cache) for e in spec.schedule] == \
        [(0, 0, False), (1, None, False), (2, None, False), (0, 1, True), (1, None, True), (2, None, True), (0, 2, True), (1, None, True),
         (2, None, True), (3, None, False)]
    assert len({e.cache_unit for e in spec.schedule}) == 10
    assert spec.pass_input.params["passes"] == 3
    _, b = _spec(CFG_B)
    assert [(e.layer, e.enters_pass) for e in b.schedule] == [(0, None), (1, None), (2, 0), (2, 1), (3, None), (4, None)]
    # without a loop there is no pass and nothing of the embedding is kept
    plain = dict(CFG_B)
    del plain["loop"]
    _, s = _spec(plain)
    assert s.pass_input is None and not s.embedding.params["keep"] and all(e.enters_pass is None for e in s.schedule)
    plain["loop"] = None
    assert _spec(plain)[1].pass_input is None
    # one pass is still a pass
    _, s = _spec(dict(CFG_B, loop=dict(start=0, stop=5, times=1)))
    assert [e.enters_pass for e in s.schedule] == [0, None, None, None, None] and not any(e.private_cache for e in s.schedule)


def test_cache_needs_and_tensor_names():
    from mini_llm_b200.cache.manager import CacheManager, PagedNeed, StateNeed
    from mini_llm_b200.parts.model import Model
    _, spec = _spec(CFG_A)
    needs = Model(spec).layer_needs()
    # the window travels with the need; key rows padded to 16-byte pieces (20 -> 24); a latent row is key and value at once
    assert needs[1] == PagedNeed(kv_heads=2, head_dim=24, v_head_dim=12, window=25)
    assert needs[2] == PagedNeed(kv_heads=1, head_dim=48, values_in_keys=True)
    assert needs[0] == StateNeed((3 * (16 * 24 + 16 + 1),), "float32") and needs[3] == StateNeed((40 * 8 + 40 + 1,), "float32")
    assert len(needs) == 10                               # four layers and six further runs of the looped ones
    cm = CacheManager(needs, page_size=8, num_pages=4, max_num_seqs=2, allocate=False)
    assert sorted(len(g.layers) for g in cm.groups) == [3, 3] and len(cm.state_layers) == 4
    for cfg in (CFG_A, CFG_B):
        _, s = _spec(cfg)
        assert {ref.canonical for _, ps in s.all_part_specs() for ref in ps.weights.values()} == set(make_tensors(cfg, 0))
    names = set(make_tensors(CFG_A, 0))
    assert {"loop.in", "loop.step", "head", "l0.mix.i.b", "l0.mix.norm", "l1.mix.talk", "l1.mix.o.b", "l2.mix.dq.norm", "l2.mix.uq",
            "l2.mix.sink", "l2.mix.g", "l2.mlp.down.b", "l2.norm2b", "final.norm"} <= names and "l3.norm2" not in names


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="mamba2"), "type must be one of"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "not a multiple of kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(mask=7), "mask must be an object"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size must be >= 1"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "at most rot_dim"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(base=0.0), "base must be positive"),
    (lambda c: c["layers"][2]["mixer"].pop("q_rank"), "q_rank must be an integer"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0.0), "gate_cap must be positive"),
    (lambda c: c["layers"][0]["mixer"].pop("vdim"), "vdim must be an integer"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind must be one of"),
    (lambda c: c["loop"].update(stop=5), "no stretch of the 4 layers"),
    (lambda c: c["loop"].update(start=3), "no stretch of the 4 layers"),
    (lambda c: c["loop"].update(times=0), "times must be >= 1"),
    (lambda c: c.update(loop=[0, 3]), "'loop' must be an object"),
    (lambda c: c.pop("residual_mult"), "missing required key 'residual_mult'"),
    (lambda c: c["embedding"].pop("scale"), "scale must be a number"),
    (lambda c: c.pop("norm"), "missing required key 'norm'"),
])
def test_config_errors(change, match):
    from mini_llm_b200.config.base import ConfigError
    cfg = copy.deepcopy(CFG_A)
    change(cfg)
    with pytest.raises(ConfigError, match=match):
        _spec(cfg)


def test_parts_refuse_what_they_cannot_do():
    from mini_llm_b200.parts.attention import MixedScoreAttention
    from mini_llm_b200.parts.embedding import TokenEmbedding
    from mini_llm_b200.parts.latent import LatentAttention
    from mini_llm_b200.parts.mlstm import MatrixMemoryMixer
    from mini_llm_b200.parts.spec import ModelSpec, PartSpec, ScheduleEntry
    with pytest.raises(ValueError, match="multiple"):
        MixedScoreAttention(8, 3, 2, 4, 4, 1.0)
    with pytest.raises(ValueError, match="sink"):
        MixedScoreAttention(8, 2, 2, 4, 4, 1.0, sink="one")
    with pytest.raises(ValueError, match="gate"):
        LatentAttention(8, 1, 4, 4, 4, 8, 1.0, 1e-5, gate="row")
    with pytest.raises(ValueError, match="positive"):
        MatrixMemoryMixer(8, 1, 4, 4, 0.0, 1e-5)
    with pytest.raises(ValueError, match="kept"):
        TokenEmbedding(8, 4, copies=2, keep=True)
    p = PartSpec("none")
    with pytest.raises(ValueError, match="enters a pass"):
        ModelSpec(8, 4, p, p, [None], p, p, schedule=[ScheduleEntry(0, enters_pass=0)])


def test_sizes_no_kernel_takes_are_refused_before_a_device_is_touched():
    from mini_llm_b200.parts.model import Model
    _, spec = _spec(config(32, 20, 1e-5, 1.0, 1.0, [layer(mlstm(1, 300, 8, 4.0), None), layer(attn(2, 1, 264, 8, 1.0, 9), None),
                                                    layer(attn(66, 1, 8, 8, 1.0, 9), None), layer(latent(1, 4, 4, 4, 4, 600, 1.0, 9.0), None)]))
    msgs = Model(spec).kernel_limits("float32")
    assert [any(w in m for m in msgs) for w in ("states of 300 x 8", "keys of 264", "66 heads", "a latent of 600")] == [True] * 4


def test_a_state_row_that_is_used_again_is_zero():
    from mini_llm_b200.cache.manager import CacheManager
    from mini_llm_b200.parts.model import Model
    _, spec = _spec(CFG_A)
    cm = CacheManager(Model(spec).layer_needs(), page_size=8, num_pages=8, max_num_seqs=1, allocate=True, device="cpu")
    cm.admit("a")
    slot = cm.slot("a")
    assert len(cm.states) == 4                            # three passes of the looped recurrence and the last layer
    for st in cm.states.values():
        st[slot].fill_(5.0)
    cm.release("a")
    cm.admit("b")
    assert cm.slot("b") == slot and all(float(st[slot].abs().max()) == 0.0 for st in cm.states.values())


def test_random_weights_folder_loads_by_name(tmp_path):
    from mini_llm_b200 import write_random_model
    from mini_llm_b200.weights.safetensors_io import Checkpoint
    out = write_random_model(CFG_A, 5, str(tmp_path / "m"), dtype="bfloat16")
    ck = Checkpoint(out)
    assert set(ck.names()) == set(make_tensors(CFG_A, 0))
    for name, t in make_tensors(CFG_A, 0).items():
        assert tuple(ck.shape(name)) == tuple(t.shape), name
    with open(tmp_path / "m" / "config.json") as f:
        assert json.load(f)["architecture"] == "Zadenex"


def test_plain_statement_against_itself():
    g = torch.Generator().manual_seed(0)
    t = make_tensors(CFG_A, 1)
    ids = torch.randint(0, CFG_A["vocab"], (60,), generator=g).tolist()
    full = P.forward(t, CFG_A, ids)
    # a prefix's logits do not depend on what follows
    assert torch.allclose(P.forward(t, CFG_A, ids[:31]), full[:31], rtol=1e-9, atol=1e-9)
    # the window and the causal edge by hand
    assert P.visible(6, 3).tolist() == [[0 <= i - j < 3 for j in range(6)] for i in range(6)]
    # mixing: a permutation hands head h the scores of another head; the transpose hands them elsewhere
    s = torch.randn(3, 2, 2, generator=g, dtype=F64)
    perm = torch.zeros(3, 3, dtype=F64)
    perm[0, 1] = perm[1, 2] = perm[2, 0] = 1.0
    assert torch.equal(P.mix_heads(s, perm), s[[1, 2, 0]]) and not torch.equal(P.mix_heads(s, perm), P.mix_heads(s, perm.T))
    # the sink: one more term of the denominator; a sink of 0 adds one
    w = P.softmax_with_sink(s, torch.tensor([0.0, -1e9, 2.0], dtype=F64))
    e = s.exp()
    assert torch.allclose(w[0], e[0] / (1.0 + e[0].sum(-1, keepdim=True))) and torch.allclose(w[1], torch.softmax(s[1], -1))
    assert torch.allclose(w[2], e[2] / (math.exp(2.0) + e[2].sum(-1, keepdim=True)))
    # a pair turned to position p and one turned to position q score by p - q alone (angles are 32-bit); neighbours are pairs
    a, b = torch.randn(1, 8, generator=g, dtype=F64), torch.randn(1, 8, generator=g, dtype=F64)
    dot = lambda i, j: float((P.rotate_pairs(a, torch.tensor([i]), 6, 50.0) * P.rotate_pairs(b, torch.tensor([j]), 6, 50.0)).sum())
    assert dot(9, 4) == pytest.approx(dot(25, 20), rel=1e-5, abs=1e-5) and abs(dot(9, 4) - dot(9, 5)) > 1e-3
    r = P.rotate_pairs(a, torch.tensor([1]), 2, 10.0)
    assert torch.allclose(r[0, 0], a[0, 0] * math.cos(1.0) - a[0, 1] * math.sin(1.0)) and torch.equal(r[0, 2:], a[0, 2:])
    # the memory cut in two with its state handed on equals the memory in one piece
    q, k = torch.randn(20, 2, 6, generator=g, dtype=F64), torch.randn(20, 2, 6, generator=g, dtype=F64)
    v = torch.randn(20, 2, 5, generator=g, dtype=F64)
    i, f = 3.0 * torch.randn(20, 2, generator=g, dtype=F64), -torch.rand(20, 2, generator=g, dtype=F64)
    o, S = P.memory_scan(q, k, v, i, f)
    o1, S1 = P.memory_scan(q[:7], k[:7], v[:7], i[:7], f[:7])
    o2, S2 = P.memory_scan(q[7:], k[7:], v[7:], i[7:], f[7:], S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and all(torch.allclose(x, y) for x, y in zip(S2, S))
    # the closed form without a running maximum: S = sum_t exp(sum_{s>t} f_s + i_t) k_t v_t^T; the maximum starts at zero, so
    # the denominator is max(|n . q|, 1) in these units and exp(-m) in the running ones
    wt = torch.stack([(f[t + 1:].sum(0) + i[t]).exp() for t in range(20)])
    num = torch.einsum("th,thi,thj,hi->hj", wt, k, v, q[-1])
    nq = torch.einsum("th,thi,hi->h", wt, k, q[-1])
    m = S[2]
    want = num * (-m).exp()[:, None] / (torch.maximum(nq.abs() * (-m).exp(), (-m).exp()) + 1e-6)[:, None]
    assert torch.allclose(o[-1], want)
    # all input gates far below zero: the maximum stays at what the forget gates leave of zero, not at the input gate
    _, (_, _, m) = P.memory_scan(q, k, v, i - 50.0, 0.0 * f)
    assert float(m.abs().max()) == 0.0
    # the gates are capped, and the forget gate's logarithm is never positive
    hh = 100.0 * torch.randn(9, 4, generator=g, dtype=F64)
    gi, gf = P.memory_gates(hh, dict(i=torch.randn(2, 4, generator=g, dtype=F64), f=torch.randn(2, 4, generator=g, dtype=F64),
                                     **{"i.b": torch.zeros(2, dtype=F64), "f.b": torch.zeros(2, dtype=F64)}), dict(gate_cap=3.0))
    assert float(gi.abs().max()) <= 3.0 and float(gf.max()) < 0.0 and float(gf.min()) >= -3.1
    # the order of the runs
    assert P.layer_runs(dict(layers=[0] * 5, loop=dict(start=1, stop=3, times=2))) == \
        [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]
    # every pass re-reads the embedded rows: with W = [0 | I] and no step the looped layer sees x0 again
    D = 4
    x, x0 = torch.randn(3, D, generator=g, dtype=F64), torch.randn(3, D, generator=g, dtype=F64)
    assert torch.equal(P.enter_pass(x, x0, torch.cat([torch.zeros(D, D, dtype=F64), torch.eye(D, dtype=F64)], 1), torch.zeros(D, dtype=F64)), x0)
