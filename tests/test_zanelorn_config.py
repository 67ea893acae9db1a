"""Zanelorn without a GPU: the configuration reader and its errors, the model description (joins, side input, cache needs, tensor
names), kept pages, the random-weights folder, and the plain statement against itself."""
import copy
import json
import math

import pytest
import torch

import plain_zanelorn as P
from zanelorn_models import CFG_A, CFG_B, attn, config, dense, layer, make_tensors, moe, parallel, retention

F64 = torch.float64


def _spec(cfg):
    import mini_llm_b200  # noqa: F401
    from mini_llm_b200.config.base import config_from_dict, get_architecture
    c = config_from_dict(cfg)
    return c, get_architecture(c.architecture).build_spec(c)


def test_every_size_is_read_per_layer():
    c, spec = _spec(CFG_A)
    assert c.architecture == "Zanelorn"
    assert (c.vocab, c.width, c.norm_eps, c.embedding_scale, c.residual_mult, c.side_dim) == (97, 64, 1e-5, 1.5, 0.7, 12)
    a, b, d, e = (l.mixer for l in c.layers)
    assert (a.left.heads, a.left.kv_heads, a.left.dim, a.left.vdim, a.left.scale, a.left.window, a.left.keep_first) == (6, 2, 20, 12, 0.3, 25, 5)
    assert (a.left.rot.base, a.left.rot.dims, a.left.rot.factor, e.left.rot.factor) == (100.0, 8, 3.0, 8.0)
    assert (a.right.inner, a.right.state, a.right.dt_rank, a.right.conv, a.left_scale, a.right_scale) == (48, 10, 5, 4, 0.8, 1.1)
    assert (b.heads, b.dim, b.vdim, b.decay, b.rot.base, b.rot.dims, b.rot.factor) == (3, 16, 24, [0.9, 0.97, 0.999], 1000.0, 16, None)
    assert (d.heads, d.rot.dims) == (1, 12)
    assert [l.mixer.kind for l in spec.layers] == ["parallel", "retention", "retention", "parallel"]
    assert all(l.arrangement == "output_norm" and l.mixer_norm is None and l.mixer_join.params["factor"] == 0.7 for l in spec.layers)
    assert [l.side.params["part"] for l in spec.layers] == [0, 1, 2, 3] and spec.token_table.params == dict(vocab_size=97, parts=4, dim=12)
    assert spec.layers[2].ff is None and spec.layers[2].ff_join is None and r"^l2\.norm2$" in spec.ignored_tensors
    left, right = (x["params"] for x in spec.layers[0].mixer.params["branches"])
    assert (left["window"], left["keep_first"], left["head_norm"], left["out_gate"], left["bias"], left["rot_interleaved"]) == (25, 5, "weighted", True, True, False)
    assert right["conv_taps"] == 4 and spec.layers[3].mixer.params["scales"] == [1.2, -0.6]
    f = spec.layers[0].ff.params
    assert (f["num_experts"], f["identity"], f["top"], f["limit"], f["shared_size"], f["shared_limit"], f["alpha"]) == (7, 3, 2, 1.5, 40, 2.5, 1.702)
    assert f["correction"] and not f["renorm"] and f["shared_gate"]
    f = spec.layers[1].ff.params
    assert (f["activation"], f["bias"], f["inner_size"]) == ("gelu_erf", False, 72)
    assert spec.embedding.params["scale"] == 1.5 and spec.embedding.params["act_copy"] and spec.head.kind == "linear"
    c, spec = _spec(CFG_B)
    assert c.layers[2].mixer.left.window is None and c.layers[2].mixer.left.keep_first == 0
    assert spec.layers[0].ff.params["shared_size"] is None and not spec.layers[0].ff.params["shared_gate"]
    assert spec.layers[1].ff.params["identity"] == 0


def test_optional_keys_may_be_null_or_absent():
    cfg = copy.deepcopy(CFG_A)
    cfg["layers"][0]["mixer"]["left"]["mask"] = None
    cfg["layers"][3]["mixer"]["left"]["mask"].pop("keep_first")
    cfg["layers"][0]["mixer"]["left"]["rot"]["scaling"] = None
    cfg["layers"][0]["mlp"]["router"].pop("identity")
    cfg["layers"][0]["mlp"]["shared"] = None
    cfg["layers"][1].pop("mlp")
    c, spec = _spec(cfg)
    a, e = c.layers[0].mixer.left, c.layers[3].mixer.left
    assert (a.window, a.keep_first, a.rot.factor, e.window, e.keep_first) == (None, 0, None, 60, 0)
    assert c.layers[0].mlp.identity == 0 and c.layers[0].mlp.shared_ff is None and spec.layers[1].ff is None
    assert "shared.sg" not in spec.layers[0].ff.weights


def test_cache_needs_and_tensor_names():
    from mini_llm_b200.cache.manager import CacheManager, PagedNeed, StateNeed
    from mini_llm_b200.parts.model import Model
    _, spec = _spec(CFG_A)
    needs = Model(spec).layer_needs()
    # window and kept tokens travel with the need; key rows padded to 16-byte pieces (20 -> 24); a state beside the pages
    assert needs[0] == [PagedNeed(kv_heads=2, head_dim=24, v_head_dim=12, window=25, keep_first=5), StateNeed((48 * 10 + 3 * 48,), "float32")]
    assert needs[1] == StateNeed((3 * 16 * 24,), "float32") and needs[2] == StateNeed((40 * 8,), "float32")
    cm = CacheManager(needs, page_size=8, num_pages=4, max_num_seqs=2, allocate=False)
    assert len(cm.groups) == 2 and len(cm.state_layers) == 4
    for cfg in (CFG_A, CFG_B):
        _, s = _spec(cfg)
        assert {ref.canonical for _, ps in s.all_part_specs() for ref in ps.weights.values()} == set(make_tensors(cfg, 0))
        m = Model(s)
        for label, ps in s.all_part_specs():
            assert set(m.part(label).param_specs()) == set(ps.weights), label
        assert not m.kernel_limits("bfloat16") and not m.kernel_limits("float32")


def test_pages_with_kept_tokens_stay_and_the_rest_goes_back():
    from mini_llm_b200.cache.manager import RELEASED, CacheManager, PagedNeed
    for keep, stays in ((0, 0), (1, 1), (4, 1), (5, 2), (9, 3)):
        cm = CacheManager({0: PagedNeed(kv_heads=1, head_dim=8, window=6, keep_first=keep)}, page_size=4, num_pages=16, max_num_seqs=2, allocate=False)
        cm.admit("a")
        done = 0
        for n in (3, 2, 7, 1, 1, 10, 4, 1, 20):
            assert cm.reserve("a", n)
            cm.commit("a", n)
            done += n
            first = max(0, done - 6 + 1) // 4                # first page that a later query's window can touch
            tab = cm.table("a", 0)
            for i, p in enumerate(tab):
                assert (p != RELEASED) == (i < stays or i >= first), (keep, done, i)
            cm.check()
        cm.release("a")
        assert cm.num_free_pages() == 16


@pytest.mark.parametrize("change,match", [
    (lambda c: c["layers"][0].update(type="mlstm"), "type must be one of"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=4), "not a multiple of kv_heads"),
    (lambda c: c["layers"][0]["mixer"]["left"].update(mask=7), "mask must be an object"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0), "size must be >= 1"),
    (lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first must be >= 0"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=7), "must be even"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=22), "at most dim"),
    (lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].update(factor=0.0), "factor must be positive"),
    (lambda c: c["layers"][0]["mixer"].pop("right"), "right must be an object"),
    (lambda c: c["layers"][0]["mixer"]["right"].pop("dt_rank"), "dt_rank must be an integer"),
    (lambda c: c["layers"][0]["mixer"].pop("left_scale"), "left_scale must be a number"),
    (lambda c: c["layers"][1]["mixer"].update(decay=[0.9, 0.9]), "list of 3 numbers"),
    (lambda c: c["layers"][1]["mixer"].pop("vdim"), "vdim must be an integer"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(base=0.0), "base must be positive"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind must be one of"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=11), "top=11 of 7"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(limit=0), "limit must be positive"),
    (lambda c: c["layers"][0]["mlp"]["shared"].pop("limit"), "limit must be a number"),
    (lambda c: c["layers"][0]["mlp"].pop("router"), "router must be an object"),
    (lambda c: c.pop("token_side"), "missing required key 'token_side'"),
    (lambda c: c.pop("residual_mult"), "missing required key 'residual_mult'"),
    (lambda c: c["embedding"].pop("scale"), "scale must be a number"),
    (lambda c: c["norm"].update(eps=0), "eps must be positive"),
    (lambda c: c.update(layers=[]), "non-empty list"),
])
def test_config_errors(change, match):
    from mini_llm_b200.config.base import ConfigError
    cfg = copy.deepcopy(CFG_A)
    change(cfg)
    with pytest.raises(ConfigError, match=match):
        _spec(cfg)


def test_parts_refuse_what_they_cannot_do():
    from mini_llm_b200.parts.attention import RotaryAttention
    from mini_llm_b200.parts.embedding import TokenEmbedding
    from mini_llm_b200.parts.moe import MoEFeedForward
    from mini_llm_b200.parts.retention import RetentionMixer
    from mini_llm_b200.parts.rotary import rotary_table
    from mini_llm_b200.parts.side import SideTable, TokenSideBranch
    from mini_llm_b200.parts.spec import LayerSpec, ModelSpec, PartSpec
    with pytest.raises(ValueError, match="decays"):
        RetentionMixer(8, 2, 4, 4, [0.5], 1e-5)
    with pytest.raises(ValueError, match="rot_dims"):
        RetentionMixer(8, 1, 4, 4, [0.5], 1e-5, rot_dims=6)
    with pytest.raises(ValueError, match="not both"):
        RotaryAttention(8, 1, 1, 8, 8, 1.0, qk_norm=True, head_norm="weighted")
    with pytest.raises(ValueError, match="keep_first"):
        RotaryAttention(8, 1, 1, 8, 8, 1.0, keep_first=-1)
    with pytest.raises(ValueError, match="no groups"):
        MoEFeedForward(8, 4, 1, 8, groups=2, correction=True)
    with pytest.raises(ValueError, match="not there"):
        MoEFeedForward(8, 4, 1, 8, shared_gate=True)
    with pytest.raises(ValueError, match="top 6"):
        MoEFeedForward(8, 4, 6, 8, identity=1)
    with pytest.raises(ValueError, match="act_copy"):
        TokenEmbedding(8, 4, copies=2, act_copy=True)
    with pytest.raises(ValueError, match="side branch"):
        TokenSideBranch(8, 4, 3).attach(SideTable(5, 3, 4))
    with pytest.raises(ValueError, match="positive factor"):
        rotary_table(8, 10.0, {"factor": 0.0})
    p = PartSpec("none")
    with pytest.raises(ValueError, match="token_table"):
        ModelSpec(8, 8, p, p, [LayerSpec(p, None, None, None, side=p)], p, p)


def test_random_weights_folder_loads_by_name(tmp_path):
    import mini_llm_b200 as m
    from mini_llm_b200.weights.safetensors_io import Checkpoint
    d = str(tmp_path / "w")
    m.write_random_model(CFG_A, 1, d, dtype="bfloat16")
    ck = Checkpoint(d)
    want = make_tensors(CFG_A, 0)
    assert set(ck.names()) == set(want)
    for n in ck.names():
        assert tuple(ck.shape(n)) == tuple(want[n].shape), n
    ck.close()
    cfg = json.load(open(tmp_path / "w" / "config.json"))
    assert cfg["architecture"] == "Zanelorn" and _spec(cfg)[0].layers[1].mixer.decay == [0.9, 0.97, 0.999]


def test_linear_scaling_of_the_frequencies():
    from mini_llm_b200.parts.rotary import rotary_table
    plain, one = rotary_table(12, 50.0)
    f, size = rotary_table(12, 50.0, {"factor": 4.0})
    assert (one, size) == (1.0, 1.0) and all(abs(a - b / 4.0) < 1e-15 for a, b in zip(f, plain))


# ------------------------------------------------------------------------------------------- the statement against itself
def test_visible_by_hand():
    m = P.visible(9, 3, 2)
    assert [[j for j in range(9) if m[i, j]] for i in (0, 1, 2, 4, 5, 8)] == [[0], [0, 1], [0, 1, 2], [0, 1, 2, 3, 4], [0, 1, 3, 4, 5], [0, 1, 6, 7, 8]]
    assert torch.equal(P.visible(5, None), torch.tril(torch.ones(5, 5, dtype=torch.bool)))
    assert torch.equal(P.visible(6, 2, 6), P.visible(6, None))


def test_rotation_keeps_lengths_and_sees_distances_only():
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 1, 10, dtype=F64, generator=g), torch.randn(1, 1, 10, dtype=F64, generator=g)

    def at(x, p, f=1.0):
        return P.rotate_halves(x, torch.tensor([p]), 8, 100.0, f)[0, 0]
    assert abs(at(q, 77).norm() - q.norm()) < 1e-12 and torch.equal(at(q, 77)[8:], q[0, 0, 8:]) and torch.equal(at(q, 0), q[0, 0])
    assert abs(at(q, 40) @ at(k, 33) - at(q, 17) @ at(k, 10)) < 1e-5
    assert abs(at(q, 4) @ at(k, 2) - at(q, 8, 2.0) @ at(k, 4, 2.0)) < 1e-6        # half the frequency, twice the distance


def test_retention_in_closed_form_and_cut_in_two():
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(9, 2, d, dtype=F64, generator=g) for d in (4, 4, 3))
    a = [0.5, 0.9]
    o, S = P.retention_scan(q, k, v, a)
    for h in range(2):
        w = torch.tensor([[a[h] ** (i - j) if j <= i else 0.0 for j in range(9)] for i in range(9)], dtype=F64)
        assert (o[:, h] - ((q[:, h] @ k[:, h].T) * w) @ v[:, h]).abs().max() < 1e-12
    o1, S1 = P.retention_scan(q[:4], k[:4], v[:4], a)
    o2, S2 = P.retention_scan(q[4:], k[4:], v[4:], a, S1)
    assert torch.equal(torch.cat([o1, o2]), o) and torch.equal(S2, S)


def test_selective_scan_cut_in_two_and_its_limits():
    g = torch.Generator().manual_seed(2)
    x, dt, A = torch.randn(8, 3, dtype=F64, generator=g), torch.rand(8, 3, dtype=F64, generator=g), -torch.rand(3, 4, dtype=F64, generator=g)
    B, C, D = torch.randn(8, 4, dtype=F64, generator=g), torch.randn(8, 4, dtype=F64, generator=g), torch.randn(3, dtype=F64, generator=g)
    y, S = P.selective_scan(x, dt, A, B, C, D)
    y1, S1 = P.selective_scan(x[:5], dt[:5], A, B[:5], C[:5], D)
    y2, S2 = P.selective_scan(x[5:], dt[5:], A, B[5:], C[5:], D, S1)
    assert torch.equal(torch.cat([y1, y2]), y) and torch.equal(S2, S)
    y, _ = P.selective_scan(x, dt, A * 1e6, B, C, D)         # forgets at once: the current token only
    assert (y - (dt * x * (B * C).sum(1, keepdim=True) + D * x)).abs().max() < 1e-9
    y, _ = P.selective_scan(x, dt, A * 0.0, B, C, D)         # keeps everything
    assert (y[-1] - ((dt * x)[:, :, None] * B[:, None, :]).sum(0) @ C[-1] - D * x[-1]).abs().max() < 1e-12


def test_convolution_by_hand():
    x = torch.tensor([[1.0], [10.0], [100.0]], dtype=F64)
    y = P.causal_conv(x, torch.tensor([[3.0, 2.0, 1.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert y.flatten().tolist() == [1.5, 12.5, 123.5]


def test_the_choice_is_corrected_and_the_weights_are_not():
    z = torch.log(torch.tensor([[0.5, 0.3, 0.15, 0.05]], dtype=F64))
    idx, w = P.choose(z, torch.zeros(4, dtype=F64), 2)
    assert idx.tolist() == [[0, 1]] and torch.allclose(w, torch.tensor([[0.5, 0.3]], dtype=F64))
    idx, w = P.choose(z, torch.tensor([0.0, -0.2, 0.0, 0.4], dtype=F64), 2)
    assert sorted(idx[0].tolist()) == [0, 3] and abs(float(w.sum()) - 0.55) < 1e-12


def test_identity_experts_give_the_input_back():
    D = 6
    g = torch.Generator().manual_seed(3)
    h = torch.randn(2, D, dtype=F64, generator=g)
    w = {"router": torch.zeros(3, D, dtype=F64), "correction": torch.tensor([-1.0, 0.0, 1.0], dtype=F64)}
    y = P.moe(h, w, dict(router=dict(experts=1, top=2), expert=dict(limit=1.0), shared=None))
    assert torch.allclose(y, h * 2.0 / 3.0)                 # two of three equal scores, both identity


def test_clamps_are_one_sided_for_the_gate_and_two_sided_for_the_other():
    one = torch.eye(1, dtype=F64)

    def f(x, gate, up):
        return float(P.clamped_expert(torch.tensor([[x]], dtype=F64), gate * one, up * one, one, 2.0))

    def y(g, u):
        return g / (1.0 + math.exp(-1.702 * g)) * (u + 1.0)
    assert abs(f(5.0, 1.0, 0.1) - y(2.0, 0.5)) < 1e-12 and abs(f(-5.0, 1.0, 0.1) - y(-5.0, -0.5)) < 1e-12
    assert abs(f(5.0, 0.1, 1.0) - y(0.5, 2.0)) < 1e-12 and abs(f(-5.0, 0.1, 1.0) - y(-0.5, -2.0)) < 1e-12


def test_a_sequence_does_not_see_its_future_and_layers_read_their_own_side_columns():
    t = make_tensors(CFG_A, 2)
    ids = torch.randint(0, 97, (40,), generator=torch.Generator().manual_seed(0)).tolist()
    full = P.forward(t, CFG_A, ids)
    assert (P.forward(t, CFG_A, ids[:23]) - full[:23]).abs().max() < 1e-10
    base, other = [], []
    P.forward(t, CFG_A, ids, trace=base)
    t2 = dict(t)
    t2["side.embed"] = t["side.embed"].clone()
    t2["side.embed"][:, 2 * 12:3 * 12] += 1.0               # the third layer's columns
    P.forward(t2, CFG_A, ids, trace=other)
    assert torch.equal(base[0], other[0]) and torch.equal(base[1], other[1]) and not torch.equal(base[2], other[2])


def test_small_models_build_on_the_host():
    cfg = config(24, 30, 1e-5, 1.0, 0.5, 4, [layer(parallel(attn(2, 1, 8, 4, 0.5, 10.0, window=3, keep=1), 8, 4, 2, 2), moe(2, 1, 1, 8, 1.0)),
                                             layer(retention(1, 4, 4, (0.5,), 10.0), dense(8))])
    _, spec = _spec(cfg)
    assert len(spec.layers) == 2 and len(P.greedy(make_tensors(cfg, 0), cfg, [1, 2], 3)) == 3
