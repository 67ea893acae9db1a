"""Zanelorn through the engine (ModelRunner, the cache manager, the scheduler, LLM.generate, bin/trace_run) against the plain
float64 statement in tests/plain_zanelorn.py, on small models made here with weights that make faults show."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_zanelorn as P
from helpers import ROOT, Replay, random_ids, write_model
from zanelorn_models import CONFIGS, PAGE, attn, config, dense, layer, make_tensors, moe, parallel, retention

pytestmark = pytest.mark.gpu


def oracle(tensors, cfg, ids, dtype):
    return P.forward(tensors, cfg, ids, store=P.to_bf16 if dtype == "bfloat16" else P._keep).numpy()


def close(got, want, dtype, what):
    """Row by row: relative error at most 2e-5 in float32.  bfloat16: the median row within 1e-2 and all but one in fifty (and
    one) within 3e-2: where two experts' choice scores nearly tie, a value on the other side of a rounding edge picks the other
    one (the plain statement in float32 instead of float64 differs from itself by up to 4e-2 in such a row when both round to
    bfloat16 where the engine does, and by 1.4e-2 in the others)."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    assert got.shape == want.shape and np.isfinite(got).all(), what
    err = np.linalg.norm(got - want, axis=1) / np.maximum(np.linalg.norm(want, axis=1), 1e-12)
    if dtype == "float32":
        assert err.max() <= 2e-5, f"{what}: row {err.argmax()}: relative error {err.max():.3e}"
        return
    over = int((err > 3e-2).sum())
    assert np.median(err) <= 1e-2 and over <= 1 + len(err) // 50, f"{what}: worst {np.sort(err)[-5:]}, median {np.median(err):.3e}"


def runner_for(folder, which, dtype, pages=160, seqs=4, graphs=False):
    from mini_llm_b200.config.base import EngineConfig
    from mini_llm_b200.engine.runner import ModelRunner
    return ModelRunner(folder, EngineConfig(dtype=dtype, page_size=PAGE[which], num_pages=pages, max_num_seqs=seqs,
                                            use_cuda_graphs=graphs))


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for which in CONFIGS:
        tensors = make_tensors(CONFIGS[which], seed=3)
        folder = write_model(str(tmp_path_factory.mktemp("zanelorn_" + which)), CONFIGS[which], tensors, torch.bfloat16)
        out[which] = (folder, tensors)
    return out


def test_layers_one_by_one_in_float32(models):
    """The residual after every layer against the oracle's."""
    from mini_llm_b200 import ops
    from mini_llm_b200.engine.runner import StepEntry
    for which in CONFIGS:
        folder, tensors = models[which]
        cfg = CONFIGS[which]
        ids = random_ids(75, cfg["vocab"], 5)
        res = []
        P.forward(tensors, cfg, ids, trace=res)
        r = runner_for(folder, which, "float32")
        r.add_request("a")
        ctx = r.prepare_step([StepEntry("a", ids, [0])])
        m = r.model
        assert len(m.layers) == len(res)
        with ops.stream_scope():
            x = m.embedding.forward(ctx, m.positions)
            for i, (lay, cache) in enumerate(zip(m.layers, m._caches)):
                x = lay.arrangement(lay, x, ctx, cache)
                assert (x.double().cpu() - res[i]).abs().max() < 3e-5 * res[i].abs().max(), (which, i)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B"])
def test_whole_prompts_then_token_by_token(models, which, dtype):
    from mini_llm_b200.engine.runner import StepEntry
    folder, tensors = models[which]
    cfg = CONFIGS[which]
    n = 330                                    # many windows of every layer, past a split of keys
    ids = random_ids(n, cfg["vocab"], 7)
    want = oracle(tensors, cfg, ids, dtype)
    r = runner_for(folder, which, dtype)
    r.add_request("w")
    got = r.step([StepEntry("w", ids, list(range(n)))]).cpu().numpy()
    close(got, want, dtype, "whole")
    r.finish_request("w")
    # most of it in one step, the rest one by one: long decoding over the windows' edges, with every state carried from
    # token to token, through pages and state rows that the request before has just given back
    r.add_request("d")
    head = n - 120
    rows = [r.step([StepEntry("d", ids[:head], [0, 1, 2, head - 1])]).cpu().numpy()]
    for t in range(head, n):
        rows.append(r.step([StepEntry("d", [ids[t]], [0])]).cpu().numpy())
    close(np.concatenate(rows), want[[0, 1, 2, head - 1] + list(range(head, n))], dtype, "decode")
    r.finish_request("d")
    # from the very first token on, one by one: a single key, states that are still zero, no input for the convolution yet
    r.add_request("f")
    rows = [r.step([StepEntry("f", [ids[t]], [0])]).cpu().numpy() for t in range(40)]
    close(np.concatenate(rows), want[:40], dtype, "first tokens")
    r.finish_request("f")
    r.cache.check()
    assert r.cache.num_live == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B"])
def test_portions_of_many_sizes(models, which, dtype):
    """Cuts of one and two tokens, mid-page, mid-window, among the kept tokens, exactly at a window's edge and one token to
    either side, inside the convolution's reach, and at the edges of the recurrences' chunks of 16 tokens."""
    from mini_llm_b200.engine.runner import StepEntry
    folder, tensors = models[which]
    cfg = CONFIGS[which]
    n = 290
    ids = random_ids(n, cfg["vocab"], 11)
    want = oracle(tensors, cfg, ids, dtype)
    r = runner_for(folder, which, dtype)
    for cuts in ([2, 2, 3, 64, 1, 31, 2, 17, 33, 2, 1, 1, 2, 129], [24, 13, 27, 36, 99, 1, 90], [2] * 100 + [90],
                 [25, 2, 43, 1, 69, 2, 71, 77], [16, 16, 15, 17, 32, 1, 193]):
        assert sum(cuts) == n
        r.add_request("p")
        rows, at = [], 0
        for c in cuts:
            rows.append(r.step([StepEntry("p", ids[at:at + c], list(range(c)))]).cpu().numpy())
            at += c
        close(np.concatenate(rows), want, dtype, f"portions {cuts[:4]}")
        r.finish_request("p")
    r.cache.check()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("which", ["A", "B"])
@pytest.mark.parametrize("graphs", [False, True])
def test_unequal_requests_batched_with_pages_used_again(models, which, dtype, graphs):
    """Five requests through three places and a pool that cannot hold them all at once: portions beside single tokens,
    requests that sit a step out, pages given back (also by the window, while a request runs) and state rows taken by the next
    request.  Every row equals the request run alone (the oracle)."""
    from mini_llm_b200.engine.runner import StepEntry
    folder, tensors = models[which]
    cfg = CONFIGS[which]
    lens = {"a": 90, "b": 13, "c": 121, "d": 2, "e": 64}
    ids = {k: random_ids(n, cfg["vocab"], 20 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: oracle(tensors, cfg, v, dtype) for k, v in ids.items()}
    plan = {"a": [30, 2, 1, 1, 40, 1, 1, 14], "b": [2, 1, 1, 9], "c": [64, 1, 0, 50, 2, 1, 1, 1, 1], "d": [2],
            "e": [1, 1, 1, 1, 1, 59]}
    ps = PAGE[which]
    r = runner_for(folder, which, dtype, pages=(90 + 16 + 121 + 64) // ps + 6, seqs=3, graphs=graphs)
    waiting, live, at, got = ["a", "b", "c", "d", "e"], [], {k: 0 for k in lens}, {k: [] for k in lens}
    while waiting or live:
        while waiting and len(live) < 3:
            k = waiting.pop(0)
            r.add_request(k)
            live.append(k)
        entries = []
        for k in live:
            c = plan[k].pop(0)
            if c:
                entries.append(StepEntry(k, ids[k][at[k]:at[k] + c], list(range(c))))
        out = r.step(entries).cpu().numpy()
        o = 0
        for e in entries:
            c = len(e.tokens)
            got[e.req].append(out[o:o + c])
            o += c
            at[e.req] += c
        for k in list(live):
            if not plan[k]:
                r.finish_request(k)
                live.remove(k)
        r.cache.check()
    for k in lens:
        close(np.concatenate(got[k]), want[k], dtype, f"request {k}")
    assert r.cache.num_live == 0
    assert all(g.allocator.num_in_use == 0 for g in r.cache.groups)


def test_a_request_alone_and_in_a_batch(models):
    """What else is in the step changes nothing beyond rounding (a product of more rows may take another kernel)."""
    from mini_llm_b200.engine.runner import StepEntry
    for which in CONFIGS:
        folder, _ = models[which]
        cfg = CONFIGS[which]
        a, b, c = (random_ids(n, cfg["vocab"], 70 + n) for n in (37, 9, 64))
        r = runner_for(folder, which, "float32")
        r.add_request("a")
        alone = [r.step([StepEntry("a", a[:30], [29])]).clone()]
        alone += [r.step([StepEntry("a", [t], [0])]).clone() for t in a[30:]]
        r.finish_request("a")
        for k in "abc":
            r.add_request(k)
        r.step([StepEntry("c", c[:5], []), StepEntry("b", b[:3], [])])
        both = [r.step([StepEntry("b", b[3:], []), StepEntry("a", a[:30], [29]), StepEntry("c", c[5:40], [0])])[:1].clone()]
        for i, t in enumerate(a[30:]):
            both.append(r.step([StepEntry("c", [c[40 + i]], [0]), StepEntry("a", [t], [0])])[1:2].clone())
        a1, a2 = torch.cat(alone).double(), torch.cat(both).double()
        assert ((a1 - a2).norm(dim=1) / a1.norm(dim=1)).max() < 2e-5, which


def test_state_rows_that_are_used_again_start_from_zero(models):
    """One place, three requests one after the other: the second and third find every layer's states of the one before in their
    slot and must not see them."""
    from mini_llm_b200.engine.runner import StepEntry
    for which in CONFIGS:
        folder, tensors = models[which]
        cfg = CONFIGS[which]
        r = runner_for(folder, which, "float32", seqs=1)
        for i, n in enumerate((50, 21, 34)):
            ids = random_ids(n, cfg["vocab"], 90 + i)
            r.add_request(i)
            got = [r.step([StepEntry(i, ids[:n - 5], list(range(n - 5)))]).cpu().numpy()]
            got += [r.step([StepEntry(i, [t], [0])]).cpu().numpy() for t in ids[n - 5:]]
            close(np.concatenate(got), oracle(tensors, cfg, ids, "float32"), "float32", f"request {i} in the only slot")
            r.finish_request(i)


def test_pages_between_the_kept_tokens_and_the_window_go_back_while_a_request_runs(tmp_path):
    """Windows of 40 and 11 kept tokens over pages of 8: what no query can see any more returns to the pool, the two pages with
    kept tokens stay, so a pool far smaller than the sequence carries it, and the rows stay right."""
    from mini_llm_b200.config.base import EngineConfig
    from mini_llm_b200.engine.runner import ModelRunner, StepEntry
    cfg = config(48, 61, 1e-5, 2.0, 0.6, 8, [layer(parallel(attn(2, 1, 16, 16, 0.5, 100.0, window=40, keep=11), 16, 4, 2, 4), dense(32)),
                                             layer(retention(2, 8, 16, (0.9, 0.99), 10.0), None),
                                             layer(parallel(attn(4, 2, 8, 8, 0.6, 1e3, window=40, keep=11), 24, 8, 3, 2), None)])
    tensors = make_tensors(cfg, 8)
    folder = write_model(str(tmp_path / "m"), cfg, tensors, torch.bfloat16)
    n = 400
    ids = random_ids(n, cfg["vocab"], 2)
    want = oracle(tensors, cfg, ids, "float32")
    r = ModelRunner(folder, EngineConfig(dtype="float32", page_size=8, num_pages=20, max_num_seqs=1, use_cuda_graphs=False))
    r.add_request("a")
    rows, at = [], 0
    for c in [50, 30, 47, 1, 1, 1, 70] + [1] * 200:
        rows.append(r.step([StepEntry("a", ids[at:at + c], list(range(c)))]).cpu().numpy())
        at += c
        # the window's 40 tokens span at most six pages, the kept ones two
        assert all(g.allocator.num_in_use <= 8 and min(g.tables["a"][:2]) >= 0 for g in r.cache.groups)
    assert at == n
    close(np.concatenate(rows), want, "float32", "a pool smaller than the sequence")
    r.finish_request("a")
    r.cache.check()
    assert all(g.allocator.num_in_use == 0 for g in r.cache.groups)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(models, dtype):
    """LLM.generate (scheduler, prompt portions under a small token budget, several requests decoding together, places used
    again) gives the oracle's greedy tokens; where the oracle's two best logits are closer than the comparison rule allows,
    either token is taken and the oracle follows the engine."""
    from mini_llm_b200 import LLM, SamplingParams
    folder, tensors = models["A"]
    cfg = CONFIGS["A"]
    prompts = [random_ids(n, cfg["vocab"], 40 + n) for n in (33, 5, 70, 1, 18)]
    new = 12
    llm = LLM(folder, dtype=dtype, page_size=8, num_pages=60, max_num_seqs=3, max_num_batched_tokens=48, prefill_chunk=32)
    outs = llm.generate(prompts, SamplingParams(max_new_tokens=new, ignore_eos=True))
    margin = 1e-3 if dtype == "float32" else 0.25
    for p, out in zip(prompts, outs):
        assert len(out) == new
        seq = list(p)
        for tok in out:
            logits = oracle(tensors, cfg, seq, dtype)[-1]
            best = int(np.argmax(logits))
            assert tok == best or logits[best] - logits[tok] < margin, (len(p), len(seq))
            seq.append(tok)
    assert llm.runner.cache.num_live == 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_with_graphs(models, dtype, tmp_path):
    """bin/trace_run on a Zanelorn folder: config.json picks the model class; steps that come back are replayed as CUDA
    graphs."""
    folder, tensors = models["B"]
    cfg = CONFIGS["B"]
    ids = {k: random_ids(n, cfg["vocab"], 60 + i) for i, (k, n) in enumerate({"p": 70, "q": 45}.items())}
    want = {k: oracle(tensors, cfg, v, dtype) for k, v in ids.items()}
    os.makedirs(tmp_path / "out")
    rp = Replay(folder, dtype, str(tmp_path / "out"), 192, page_size=PAGE["B"])
    got, at = {k: [] for k in ids}, {k: 0 for k in ids}
    plan = [[("p", 40), ("q", 30)]] + [[("p", 1), ("q", 1)]] * 15 + [[("p", 15)]]
    for step in plan:
        entries = [(k, ids[k][at[k]:at[k] + c], list(range(c))) for k, c in step]
        end = [k for k, c in step if at[k] + c == len(ids[k])]
        out = rp.step(entries, end)
        o = 0
        for k, c in step:
            got[k].append(out[o:o + c])
            o += c
            at[k] += c
    assert rp.close() == 0
    assert rp.stats["graph_replays"] >= 13
    for k in ids:
        close(np.concatenate(got[k]), want[k], dtype, f"replayed request {k}")


def test_long_contexts_with_a_key_far_back(tmp_path):
    """1,500 tokens: an attention that sees everything (several splits of keys), a window of 700 with 300 kept tokens (more than a
    split), a window of one tile with one kept token, retention heads that still carry the first tokens; whole, then in
    portions and single tokens, at rows on both sides of every edge."""
    from mini_llm_b200.config.base import EngineConfig
    from mini_llm_b200.engine.runner import ModelRunner, StepEntry
    cfg = config(72, 131, 1e-5, 2.0, 0.5, 8, [
        layer(parallel(attn(3, 3, 16, 16, 0.5, 1e4), 32, 8, 4, 4), dense(48)),
        layer(parallel(attn(6, 3, 32, 32, 0.4, 1e5, factor=4.0, window=700, keep=300), 24, 16, 8, 3), None),
        layer(retention(2, 32, 48, (0.999, 0.9999), 10000.0), dense(56)),
        layer(parallel(attn(4, 1, 16, 16, 0.5, 500.0, window=64, keep=1), 16, 4, 2, 2), None)])
    tensors = make_tensors(cfg, 11)
    folder = write_model(str(tmp_path / "long"), cfg, tensors, torch.bfloat16)
    n = 1500
    ids = random_ids(n, cfg["vocab"], 1)
    rows = [0, 1, 63, 64, 65, 255, 256, 257, 299, 300, 511, 512, 699, 700, 701, 999, 1000, 1001, 1023, 1024, 1025, 1279, 1280, 1399, 1400, 1499]
    for dtype in ("float32", "bfloat16"):
        want = oracle(tensors, cfg, ids, dtype)
        r = ModelRunner(folder, EngineConfig(dtype=dtype, page_size=16, num_pages=200, max_num_seqs=2))
        r.add_request("w")
        close(r.step([StepEntry("w", ids, rows)]).cpu().numpy(), want[rows], dtype, "whole")
        r.finish_request("w")
        r.add_request("p")
        got, at = [], 0
        cuts = [690, 9, 2, 322, 2, 255, 200] + [1] * 20
        for c in cuts:
            got.append(r.step([StepEntry("p", ids[at:at + c], [c - 1])]).cpu().numpy()[0])
            at += c
        close(np.stack(got), want[np.cumsum(cuts) - 1], dtype, "portions and single tokens")
        assert r.graph_replays >= 15


def test_sizes_that_happen_to_be_one_or_equal(tmp_path):
    """One head, windows of one and two positions, no kept token or more than the window, no rotated entries, states of one
    number, a convolution of one tap, one expert, all of them chosen, only identity experts beside one, factors of one (and a
    negative one) on the embedding, the residual and the branches, a side input of one column, a model of one kind of layer
    only: nothing rests on two sizes being different or larger than 1."""
    from mini_llm_b200.config.base import EngineConfig
    from mini_llm_b200.engine.runner import ModelRunner, StepEntry
    a = config(40, 53, 1e-5, 1.0, 1.0, 1, [
        layer(parallel(attn(1, 1, 8, 8, 1.0, 10.0, dims=0, factor=1.0, window=1, keep=0), 1, 1, 1, 1, scales=(1.0, 1.0)), moe(1, 0, 1, 8, 1.0)),
        layer(parallel(attn(2, 2, 8, 4, 0.7, 3.0, dims=2, factor=1.0, window=2, keep=9), 8, 8, 8, 2, scales=(1.0, -1.0)), moe(1, 3, 4, 8, 0.5, (8, 0.5)))])
    b = config(32, 40, 1e-6, -0.75, 0.5, 32, [layer(retention(1, 1, 1, (1.0,), 10.0, dims=0), dense(32)), layer(retention(4, 8, 8, (0.0, 0.5, 0.5, 1.0), 3.0), None),
                                              layer(retention(1, 32, 1, (0.75,), 7.0, dims=2), moe(4, 4, 8, 1, 2.0, (1, 3.0)))])
    c = config(32, 40, 1e-5, 1.0, 1.0, 4, [layer(parallel(attn(4, 4, 8, 8, 0.8, 50.0), 32, 2, 1, 8), None)])
    for name, cfg in (("a", a), ("b", b), ("c", c)):
        tensors = make_tensors(cfg, 4)
        folder = write_model(str(tmp_path / name), cfg, tensors, torch.bfloat16)
        ids = random_ids(80, cfg["vocab"], 9)
        want = oracle(tensors, cfg, ids, "float32")
        r = ModelRunner(folder, EngineConfig(dtype="float32", page_size=8, num_pages=40, max_num_seqs=2, use_cuda_graphs=False))
        r.add_request("a")
        rows = [r.step([StepEntry("a", ids[:33], list(range(33)))]).cpu().numpy()]
        for t in range(33, 80):
            rows.append(r.step([StepEntry("a", [ids[t]], [0])]).cpu().numpy())
        # a head of one entry normed to its sign, a sum that vanishes before a norm: rounding is magnified there
        err = np.linalg.norm(np.concatenate(rows) - want, axis=1) / np.linalg.norm(want, axis=1)
        assert np.median(err) < 5e-6 and err.max() < 1e-3, (name, np.sort(err)[-3:])
        r2 = ModelRunner(folder, EngineConfig(dtype="bfloat16", page_size=8, num_pages=40, max_num_seqs=2, use_cuda_graphs=False))
        r2.add_request("a")
        out = r2.step([StepEntry("a", ids, list(range(80)))]).cpu().numpy()
        assert np.isfinite(out).all()


def test_odd_sizes(tmp_path):
    """A width, head sizes, value sizes, channels, ranks, inner sizes and a vocabulary that are no multiples of 8 (rows that start
    on no 16-byte boundary), three query heads per key/value head: every product and kernel takes them, in both dtypes."""
    from mini_llm_b200.config.base import EngineConfig
    from mini_llm_b200.engine.runner import ModelRunner, StepEntry
    cfg = config(50, 77, 1e-5, 1.7, 0.6, 7, [layer(retention(2, 33, 21, (0.9, 0.99), 100.0, dims=14), dense(30)),
                                             layer(parallel(attn(9, 3, 6, 5, 0.7, 30.0, window=9, keep=3), 37, 11, 3, 4), moe(5, 1, 2, 13, 1.1, (9, 2.0))),
                                             layer(parallel(attn(3, 1, 10, 7, 0.5, 500.0, dims=4), 19, 131, 13, 3), dense(17)),
                                             layer(retention(3, 5, 7, (0.6, 0.8, 0.95), 4.0, dims=4), None)])
    tensors = make_tensors(cfg, 6)
    folder = write_model(str(tmp_path / "odd"), cfg, tensors, torch.bfloat16)
    ids = random_ids(150, cfg["vocab"], 3)
    for dtype in ("float32", "bfloat16"):
        want = oracle(tensors, cfg, ids, dtype)
        r = ModelRunner(folder, EngineConfig(dtype=dtype, page_size=8, num_pages=40, max_num_seqs=2, use_cuda_graphs=False))
        r.add_request("a")
        rows = [r.step([StepEntry("a", ids[:97], list(range(97)))]).cpu().numpy()]
        rows.append(r.step([StepEntry("a", ids[97:120], list(range(23)))]).cpu().numpy())
        for t in range(120, 150):
            rows.append(r.step([StepEntry("a", [ids[t]], [0])]).cpu().numpy())
        close(np.concatenate(rows), want, dtype, "odd sizes")


def test_command_line_with_random_weights(tmp_path):
    """bin/mini_llm: the random-weights mode writes a Zanelorn folder from a config.json; greedy tokens from the command line
    equal LLM.generate's."""
    from mini_llm_b200 import LLM, SamplingParams
    cfg_path = tmp_path / "cfg.json"
    cfg_path.write_text(json.dumps(CONFIGS["A"]))
    out_dir = tmp_path / "written"
    cli = [sys.executable, os.path.join(ROOT, "bin", "mini_llm")]
    prompts = ["5 17 3 90 9 60 4", "40 2 2 31"]
    tail = ["--dtype", "float32", "--max-new-tokens", "6", "--ignore-eos", "--max-batch-num", "2"]
    for p in prompts:
        tail += ["--prompt-ids", p]
    r = subprocess.run(cli + ["--random-config", str(cfg_path), "--seed", "7", "--write-model", str(out_dir)] + tail,
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0 and os.path.isfile(out_dir / "model.safetensors"), r.stderr[-2000:]
    lines = [l for l in r.stdout.splitlines() if l.endswith("[DONE]")]
    got = [[int(t) for t in l.replace("[DONE]", "").split()] for l in lines]
    llm = LLM(str(out_dir), dtype="float32", max_num_seqs=2)
    want = llm.generate([[int(t) for t in p.split()] for p in prompts], SamplingParams(max_new_tokens=6, ignore_eos=True))
    assert got == want


def test_sizes_no_kernel_takes_are_refused_at_construction(tmp_path):
    from mini_llm_b200.config.base import ConfigError, EngineConfig
    from mini_llm_b200.engine.runner import ModelRunner
    for mix, match in ((retention(1, 264, 8, (0.5,), 10.0), "retention"), (parallel(attn(1, 1, 8, 8, 1.0, 10.0), 8, 300, 2, 2), "mamba"),
                       (parallel(attn(1, 1, 8, 8, 1.0, 10.0), 8, 4, 2, 17), "taps")):
        cfg = config(32, 50, 1e-5, 1.0, 1.0, 4, [layer(mix, None)])
        folder = write_model(str(tmp_path / match), cfg, make_tensors(cfg, 0))
        with pytest.raises(ConfigError, match=match):
            ModelRunner(folder, EngineConfig(dtype="float32", num_pages=4))
