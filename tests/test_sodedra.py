"""Sodedra through the engine (loading, cache, state slots, scheduler, sampling) against a plain implementation of its
equations: whole prompts, portions, token by token, mixed batches, reused pages and slots, far keys, window edges, greedy
generation."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import sodedra_oracle as oracle
from femirax_common import LIMIT, TARGETS, close, error, feed, make_engine, random_tokens, write_checkpoint
from sodedra_common import CONFIGS, attention, config, delta, dense, expect, mlstm, moe, row_limits, weights_of

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding_match_the_whole_prompt(tmp_path, name, target):
    cfg, w = weights_of(name)
    toks = random_tokens(75, cfg["vocab"], 1)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target)
    lim = row_limits(cfg, w, toks, want, target[1])
    for cuts in ([75], [2, 3, 17], [16], [40, 1, 1, 1], [1], [2], [33, 2, 15, 16, 5]):
        ok, worst = close(feed(eng, "r", toks, cuts), want, lim)
        assert ok, (name, cuts, worst)
    assert len(eng.model.state.free) == 4 and eng.scheduler.block_stats(0).num_used == 0


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_layer_streams(tmp_path, name, target):
    """The residual stream behind every layer of one short prompt."""
    cfg, w = weights_of(name)
    toks = random_tokens(21, cfg["vocab"], 2)
    want = []
    oracle.forward(toks, cfg, {n: t.double() for n, t in w.items()}, want)
    eng = make_engine(tmp_path, cfg, w, target)
    from xllm_b200.models import sodedra
    got, plain = [], sodedra.residual_update

    def spy(x, y, **kw):
        r = plain(x, y, **kw)
        if x is not None:
            got.append(r[0].double().cpu().clone())
        return r

    sodedra.residual_update = spy
    try:
        from xllm_b200.api.embedding import hidden_states
        hidden_states(eng, toks)
    finally:
        sodedra.residual_update = plain
    assert len(got) == len(want)
    for g, e in zip(got, want):
        assert float((g - e).pow(2).mean().sqrt() / e.pow(2).mean().sqrt()) < (1e-5 if target[1] == "float32" else 0.03)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_mixed_batches_and_reused_pages_and_slots(tmp_path, name, target):
    """Up to four live requests of unequal progress in one batch, in a pool so small that pages and slots go round."""
    cfg, w = weights_of(name, seed=3)
    reqs = {f"q{i}": random_tokens(n, cfg["vocab"], 10 + i) for i, n in enumerate((70, 9, 41, 64, 33, 1, 50, 17))}
    want = {r: expect(cfg, w, t) for r, t in reqs.items()}
    eng = make_engine(tmp_path, cfg, w, target, num_blocks=18)       # 17 pages of 16; the requests hold 30 in all
    rng = np.random.default_rng(5)
    waiting, live, got = list(reqs), {}, {r: [] for r in reqs}
    steps = 0
    while waiting or live:
        while waiting and len(live) < 4:
            live[waiting.pop(0)] = 0
        entries = []
        for r, at in live.items():
            if len(live) > 1 and rng.random() < 0.2:
                continue                                              # left out of this step
            n = min(int(rng.choice([1, 1, 2, 3, 16, 29])), len(reqs[r]) - at)
            entries.append((r, reqs[r][at:at + n], [j for j in range(n) if rng.random() < 0.6]))
        if not entries:
            continue
        logits = eng.replay_step(entries)
        row = 0
        for r, t, ws in entries:
            for j in ws:
                got[r].append((live[r] + j, logits[row]))
                row += 1
            live[r] += len(t)
            if live[r] == len(reqs[r]):
                eng.replay_end(r)
                del live[r]
        steps += 1
    for r, rows in got.items():
        if rows:
            at = [p for p, _ in rows]
            ok, worst = close(torch.stack([x for _, x in rows]), want[r][at], row_limits(cfg, w, reqs[r], want[r], target[1])[at])
            assert ok, (r, worst)
    assert steps > 10 and len(eng.model.state.free) == 4 and eng.scheduler.block_stats(0).num_used == 0


# ------------------------------------------------------------------------------------------- far keys and window edges
WINDOW = 70


def _one_layer(layer, rank, seed=11):
    """The query of token 91 points along the key of token 92: that key's score stands out among hundreds (attention), or
    its share of a slowly decaying state does.  Coordinates 0 and 1 of the embedding belong to the two tokens."""
    cfg = config([layer], vocab=96, width=64)
    w = oracle.random_weights(cfg, rank, seed)
    w["embed"][:, :2] = 0.0
    w["embed"][92, 0] = w["embed"][91, 1] = 8.0
    w["l0.norm1"].zero_()
    return cfg, w


def _far_model(kind):
    p = "l0.mix."
    if kind == "attention":
        cfg, w = _one_layer(attention(3, 3, 24, 20, WINDOW, 8, 1.6, base=1e5), (4, 4))
        w[p + "k"][:, 0] *= 2.0
        w[p + "q"][:, 1] = w[p + "k"][:, 0]
    elif kind == "mlstm":
        cfg, w = _one_layer(mlstm(3, 24, 20, cap=16.0), (4, 4))
        w[p + "k"][:, 0] *= 2.0
        w[p + "q"][:, 1] = w[p + "k"][:, 0]
        w[p + "f.b"].fill_(14.0)                                     # forget gates within 1e-5 of one
        w[p + "f"] *= 0.2
        w[p + "i"][:, 0] = 0.4                                       # and the far token writes strongly
    else:
        # the far token's key has a channel to itself, so that no later write erases what it left
        cfg, w = _one_layer(delta(3, 3, 24, 20), (4, 4))
        own = torch.arange(3) * 24
        for n in "qk":
            w[p + n][:, :2] = 0.0
            w[p + n][own] = 0.0
            w[p + n + ".conv"].zero_()
            w[p + n + ".conv"][:, -1] = 1.0
        w[p + "k"][own, 0] = 3.0
        w[p + "q"][own, 1] = 3.0
        w[p + "b"][:, 0] = 1.0
        w[p + "dt_bias"].fill_(-14.0)                                # decays within 1e-5 of one
        w[p + "a2"] *= 0.1
    w[p + "o"] *= 6.0
    return cfg, w


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("kind", ["attention", "mlstm", "channel_delta"])
def test_far_keys(tmp_path, kind, target):
    """The last token asks for one far back: at the first places, on both sides of page borders and of the sixteen-token
    tiles of the recurrences, and at a border of the portions.  The far token must show in the answer, whether the query
    ends a prompt's portion or is decoded alone."""
    cfg, w = _far_model(kind)
    eng = make_engine(tmp_path, cfg, w, target)
    n = 300 if kind != "attention" else 90
    base = random_tokens(n, 90, 4)
    lim = LIMIT[target[1]]
    places = (0, 1, 2, 3, 15, 16, 31, 32, 33, 63, 64, 200, 287, 288, 296) if n == 300 else (21, 31, 32, 33, 47, 48, 63, 64, 80)
    for far in places:
        toks = list(base)
        toks[far] = 92                                               # ids 90.. appear nowhere else
        toks[-1] = 91
        want = expect(cfg, w, toks)[-1:]
        without = list(base)
        without[-1] = 91
        seen = error(expect(cfg, w, without)[-1:], want)
        assert seen > 2 * lim, (kind, far, seen)                     # leaving the far key out would show
        for cuts in ([n], [64, 33, 2, 200, 1], [n - 3, 3], [n - 2, 2], [n - 1, 1]):
            at, i = 0, 0
            while at < n:
                m = min(cuts[i % len(cuts)], n - at)
                got = eng.replay_step([("f", toks[at:at + m], [m - 1] if at + m == n else [])])
                at, i = at + m, i + 1
            eng.replay_end("f")
            assert error(got, want) < lim, (kind, far, cuts)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("window,d,dv", [(1, 24, 24), (2, 24, 20), (16, 64, 64), (17, 128, 128), (70, 24, 20), (128, 128, 96),
                                         (129, 128, 128)])
def test_window_edges(tmp_path, window, d, dv, target):
    """A key just inside the window shows and one just outside does not, in prompts and in decoding."""
    cfg, w = _one_layer(attention(3, 3, d, dv, window, 8, 1.0, base=1e5), (4, 4))
    p = "l0.mix."
    w[p + "k"][:, 0] *= 2.0
    w[p + "q"][:, 1] = w[p + "k"][:, 0] * (24 / d)
    w[p + "o"] *= 6.0
    eng = make_engine(tmp_path, cfg, w, target)
    n, lim = 150, LIMIT[target[1]]
    base = random_tokens(n, 90, 8)
    base[-1] = 91
    plain = expect(cfg, w, base)[-1:]
    for back in (window - 2, window - 1, window, window + 1):
        if back < 1 or back >= n:
            continue
        toks = list(base)
        toks[n - 1 - back] = 92
        want = expect(cfg, w, toks)[-1:]
        if back < window:
            assert error(plain, want) > 2 * lim
        else:
            assert error(plain, want) < 1e-9
        for cuts in ([n], [n - 1, 1], [n - 2, 2], [37]):
            got = feed(eng, "e", toks, cuts)[-1:]
            assert error(got, want) < lim, (window, back, cuts)


@pytest.mark.parametrize("target", TARGETS)
def test_first_tokens(tmp_path, target):
    """Sequences of one to five tokens, as prompts and decoded from the first on, in slots that held others."""
    cfg, w = weights_of("odd", seed=7)
    eng = make_engine(tmp_path, cfg, w, target)
    feed(eng, "old", random_tokens(60, cfg["vocab"], 3), [60])
    for n in (1, 2, 3, 4, 5):
        toks = random_tokens(n, cfg["vocab"], 20 + n)
        want = expect(cfg, w, toks)
        lim = row_limits(cfg, w, toks, want, target[1])
        for cuts in ([n], [1], [2, 1]):
            ok, worst = close(feed(eng, "s", toks, cuts), want, lim)
            assert ok, (n, cuts, worst)


@pytest.mark.parametrize("target", TARGETS)
def test_long_decoding(tmp_path, target):
    """A short prompt, then hundreds of tokens one at a time across many page borders and windows."""
    cfg, w = weights_of("odd", seed=6)
    toks = random_tokens(260, cfg["vocab"], 9)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target)
    ok, worst = close(feed(eng, "d", toks, [3] + [1] * 300), want, row_limits(cfg, w, toks, want, target[1]))
    assert ok, worst


@pytest.mark.parametrize("target", TARGETS)
def test_a_batch_does_not_change_its_members(tmp_path, target):
    """The same request alone and beside three others; first tokens of a sequence included."""
    cfg, w = weights_of("aligned", seed=8)
    reqs = [random_tokens(n, cfg["vocab"], 30 + n) for n in (1, 2, 37, 48)]
    eng = make_engine(tmp_path, cfg, w, target)
    alone = [eng.replay_step([(f"a{i}", t, list(range(len(t))))]) for i, t in enumerate(reqs)]
    for i in range(4):
        eng.replay_end(f"a{i}")
    both = eng.replay_step([(f"b{i}", t, list(range(len(t)))) for i, t in enumerate(reqs)])
    row = 0
    for t, a in zip(reqs, alone):
        want = expect(cfg, w, t)
        ok, worst = close(both[row:row + len(t)], a, row_limits(cfg, w, t, want, target[1]))
        assert ok, worst
        row += len(t)
    # all four decode in one batch, in another order, one left out
    nxt = {f"b{i}": [(7 * i + 3) % cfg["vocab"]] for i in (3, 0, 2)}
    got = eng.replay_step([(r, t, [0]) for r, t in nxt.items()])
    for j, (r, t) in enumerate(nxt.items()):
        toks = reqs[int(r[1])] + t
        want = expect(cfg, w, toks)
        ok, worst = close(got[j:j + 1], want[-1:], row_limits(cfg, w, toks, want, target[1])[-1:])
        assert ok, worst


@pytest.mark.parametrize("target", TARGETS)
def test_pages_behind_the_widest_window_return(tmp_path, target):
    """A sequence far longer than the pool lives on the pages of its window."""
    cfg, w = weights_of("odd", seed=2)
    toks = random_tokens(240, cfg["vocab"], 12)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target, num_blocks=8)        # 7 pages of 16; the widest window is 34
    ok, worst = close(feed(eng, "r", toks, [40, 1, 1, 30, 2, 25]), want, row_limits(cfg, w, toks, want, target[1]))
    assert ok, worst
    assert eng.scheduler.num_window_released_blocks > 0 and eng.scheduler.block_stats(0).num_used == 0


# ------------------------------------------------------------------------------------------- scheduler and sampling
GREEDY_TARGETS = TARGETS[:2]                                          # fp32: no near ties between two implementations


def _llm(engine):
    from xllm_b200 import LLM
    llm = LLM.__new__(LLM)
    llm.engine, llm.tokenizer, llm._workers = engine, None, None
    return llm


@pytest.mark.parametrize("target", GREEDY_TARGETS)
@pytest.mark.parametrize("policy,overlap", [("prefill_first", False), ("decode_first", False), ("decode_first", True)])
def test_greedy_generation(tmp_path, policy, overlap, target):
    """LLM.generate through the scheduler: more requests than slots, prompts cut by a small token budget."""
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("odd", seed=5)
    prompts = [random_tokens(n, cfg["vocab"], 50 + n) for n in (5, 40, 17, 1, 66, 23)]
    eng = make_engine(tmp_path, cfg, w, target, max_tokens_per_batch=24, policy=policy, enable_schedule_overlap=overlap)
    outs = _llm(eng).generate(prompts, SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))
    w64 = {n: t.double() for n, t in w.items()}
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == oracle.greedy(p, 12, cfg, w64)
    assert len(eng.model.state.free) == 4 and not eng.model.state.owner


@pytest.mark.parametrize("target", GREEDY_TARGETS)
@pytest.mark.parametrize("policy", ["prefill_first", "decode_first"])
def test_preemption_rebuilds_the_state(tmp_path, policy, target):
    """So few pages that sequences are preempted, some re-admitted in the very step that pushed them out."""
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("odd", seed=5)
    prompts = [random_tokens(n, cfg["vocab"], 70 + n) for n in (30, 45, 18, 60, 25)]
    eng = make_engine(tmp_path, cfg, w, target, num_blocks=10, max_tokens_per_batch=32, policy=policy)
    outs = _llm(eng).generate(prompts, SamplingParams(max_tokens=16, temperature=0.0, ignore_eos=True))
    w64 = {n: t.double() for n, t in w.items()}
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == oracle.greedy(p, 16, cfg, w64)
    assert eng.scheduler.num_preemptions > 0
    assert len(eng.model.state.free) == 4 and not eng.model.state.owner


@pytest.mark.parametrize("target", TARGETS)
def test_sampling_parallel_samples_and_abort(tmp_path, target):
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("recurrent_only")
    eng = make_engine(tmp_path, cfg, w, target)
    llm = _llm(eng)
    sp = SamplingParams(max_tokens=9, temperature=25.0, top_p=0.99, n=3, seed=4, ignore_eos=True)
    a, b = (llm.generate([[3, 1, 4, 1, 5]], sp)[0] for _ in range(2))
    assert [o.token_ids for o in a.outputs] == [o.token_ids for o in b.outputs]
    assert len({tuple(o.token_ids) for o in a.outputs}) > 1
    eng.add_request("gone", [5, 6, 7, 8], max_tokens=50, ignore_eos=True, n=2)
    for _ in range(3):
        eng.step()
    eng.abort("gone")
    while eng.has_unfinished():
        eng.step()
    eng.step()
    assert len(eng.model.state.free) == 4 and not eng.model.state.owner
    assert len(llm.embed([[1, 2, 3], [4, 5, 6, 7]])) == 2


@pytest.mark.gpu
def test_captured_steps_survive_larger_batches(tmp_path):
    """Graphs captured for small steps keep answering after a larger step took larger expert workspaces."""
    cfg, w = weights_of("aligned", seed=9)
    eng = make_engine(tmp_path, cfg, w, ("cuda:0", "bfloat16"))
    toks = random_tokens(40, cfg["vocab"], 5)
    first = feed(eng, "a", toks, [20] + [1] * 20)
    assert eng.runner.graph_replays > 0
    eng.replay_step([("big", random_tokens(700, cfg["vocab"], 6), [])])
    eng.replay_end("big")
    again = feed(eng, "b", toks, [20] + [1] * 20)
    assert error(again, first) < 0.02


def test_replay_program(tmp_path):
    """bin/trace_run as a process: protocol, output files, answers."""
    cfg, w = weights_of("odd", seed=12)
    model = write_checkpoint(tmp_path / "m", cfg, w)
    os.makedirs(tmp_path / "out")
    a, b = random_tokens(40, cfg["vocab"], 1), random_tokens(9, cfg["vocab"], 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [3, 19]}, {"id": "b", "tokens": b[:8], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[20:39], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[39:], "want": [0]}], "end": ["b"]}]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", model, "--dtype", "float32", "--out",
                        str(tmp_path / "out"), "--max-tokens", "128", "--device", "cpu"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    assert sorted(os.listdir(tmp_path / "out")) == ["0.f32", "2.f32"]
    V = cfg["vocab"]
    read = lambda n: torch.from_numpy(np.fromfile(tmp_path / "out" / n, dtype="<f4").reshape(-1, V))
    wa, wb = expect(cfg, w, a), expect(cfg, w, b)
    assert error(read("0.f32"), wa[[3, 19]]) < 2e-4
    assert error(read("2.f32"), torch.stack([wb[8], wa[39]])) < 2e-4


def test_configuration_is_read_from_the_checkpoint(tmp_path):
    from xllm_b200.models import load_model_args, supported_models
    cfg, w = weights_of("odd")
    args = load_model_args(write_checkpoint(tmp_path, cfg, w))
    assert args.model_type == "sodedra" and "sodedra" in supported_models() and args.sliding_window == 34
    assert args.extra["layers"][0]["mixer"]["a1"] == 5 and args.extra["layers"][0]["mixer"]["g1"] == 9
    eng = make_engine(tmp_path, cfg, w, ("cpu", "float32"))
    assert eng.model.kv_layout()[1] == (2, 2, 64) and eng.model.kv_layout()[0] is None
    # a tensor the model needs is missing: loading says so
    for gone in ("l1.mix.q.b", "l0.mix.k.conv", "l2.mlp.e4.up", "l2.mix.f.b", "l0.mlp.router"):
        w2 = dict(w)
        del w2[gone]
        with pytest.raises(KeyError):
            make_engine(tmp_path / "x", cfg, w2, ("cpu", "float32"))
    for at, change in ((1, {"type": "convolution"}), (1, {"mlp": {"kind": "sparse"}}), (2, {"mlp": moe(10, 9, 28, 1.0, (5, 3))})):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][at].update(change)
        with pytest.raises(ValueError):
            make_engine(tmp_path / "y", bad, w, ("cpu", "float32"))


def test_kernel_sources_of_the_model():
    from xllm_b200 import _build
    from xllm_b200.models import ModelArgs
    from xllm_b200.models.registry import kernel_sources_of
    names = kernel_sources_of(ModelArgs(model_type="sodedra"))
    assert set(names) <= {s.stem for s in _build.kernel_sources()} and {"delta_rule", "mlstm", "moe"} <= set(names)
