"""Lukinex through the engine (loading, cache, state slots, scheduler, sampling) against a plain implementation of its
equations: whole prompts, portions, token by token, mixed batches, reused pages and slots, far keys, window edges, greedy
generation."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import lukinex_oracle as oracle
from femirax_common import LIMIT, TARGETS, close, error, feed, make_engine, random_tokens, write_checkpoint
from lukinex_common import CONFIGS, attention, config, expect, latent, moe, parallel, rotation, row_limits, weights_of

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def idle(eng, slots=4):
    """Nothing is held any more."""
    free = eng.scheduler.block_stats(0).num_used == 0
    return free and (eng.model.state is None or (len(eng.model.state.free) == slots and not eng.model.state.owner))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding_match_the_whole_prompt(tmp_path, name, target):
    cfg, w = weights_of(name)
    toks = random_tokens(75, cfg["vocab"], 1)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target, enable_prefix_cache=False)
    lim = row_limits(cfg, w, toks, want, target[1])
    for cuts in ([75], [2, 3, 17], [16], [40, 1, 1, 1], [1], [2], [33, 2, 15, 16, 5]):
        ok, worst = close(feed(eng, "r", toks, cuts), want, lim)
        assert ok, (name, cuts, worst)
    assert idle(eng)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_layer_streams(tmp_path, name, target):
    """The residual stream behind every layer of one short prompt."""
    cfg, w = weights_of(name)
    toks = random_tokens(21, cfg["vocab"], 2)
    want = []
    oracle.forward(toks, cfg, {n: t.double() for n, t in w.items()}, want)
    eng = make_engine(tmp_path, cfg, w, target)
    from xllm_b200.models import lukinex
    got, plain = [], lukinex.LukinexLayer.forward

    def spy(self, x, *a):
        h = plain(self, x, *a)
        got.append(x.double().cpu().clone())
        return h

    lukinex.LukinexLayer.__call__ = spy
    try:
        from xllm_b200.api.embedding import hidden_states
        hidden_states(eng, toks)
    finally:
        lukinex.LukinexLayer.__call__ = plain
    assert len(got) == len(want)
    for g, e in zip(got, want):
        assert float((g - e).pow(2).mean().sqrt() / e.pow(2).mean().sqrt()) < (1e-5 if target[1] == "float32" else 0.03)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["odd", "aligned", "wide"])
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
    assert steps > 10 and idle(eng)


@pytest.mark.gpu
def test_long_prompts_expand_their_latents(tmp_path):
    """Prompts of hundreds of tokens through keys and values made from the latents, whole, behind an earlier portion and
    beside decoding requests, against the other form."""
    cfg, w = weights_of("aligned", seed=4)
    toks = random_tokens(330, cfg["vocab"], 2)
    want = expect(cfg, w, toks)
    lim = row_limits(cfg, w, toks, want, "bfloat16")
    eng = make_engine(tmp_path, cfg, w, ("cuda:0", "bfloat16"), enable_graph=False)
    from xllm_b200 import ops
    calls, plain = [], ops.ragged_prefill_attention
    ops.ragged_prefill_attention = lambda *a, **k: (calls.append(1), plain(*a, **k))[1]
    try:
        for cuts in ([330], [37, 293], [290, 1, 39]):
            ok, worst = close(feed(eng, "p", toks, cuts), want, lim)
            assert ok, (cuts, worst)
        assert len(calls) == 3                                        # one of the two latent layers has heads of 128
        short = random_tokens(20, cfg["vocab"], 3)
        eng.replay_step([("d", short[:19], [])])
        both = eng.replay_step([("d", short[19:], [0]), ("p", toks[:300], list(range(300))), ("q", toks[:9], list(range(9)))])
        assert len(calls) == 4
    finally:
        ops.ragged_prefill_attention = plain
    ws = expect(cfg, w, short)
    assert close(both[:1], ws[-1:], row_limits(cfg, w, short, ws, "bfloat16")[-1:])[0]
    assert close(both[1:301], want[:300], lim[:300])[0] and close(both[301:], want[:9], lim[:9])[0]


@pytest.mark.gpu
def test_captured_portions_and_expanded_prompts_agree(tmp_path):
    """Many heads over wide latents: small portions replay captured steps in the absorbed form, large ones run expanded."""
    cfg = config([latent(16, 128, 128, 32, 300, 0.09), latent(2, 128, 128, 16, 300, 0.09, source=0)], vocab=96, width=64)
    w = oracle.random_weights(cfg, 3)
    toks = random_tokens(330, cfg["vocab"], 2)
    want = expect(cfg, w, toks)
    lim = row_limits(cfg, w, toks, want, "bfloat16")
    eng = make_engine(tmp_path, cfg, w, ("cuda:0", "bfloat16"), enable_prefix_cache=False)
    assert eng.model.max_prefill_graph_tokens == 256 and max(eng.runner.prefill_buckets) == 256
    for cuts in ([330], [200, 130], [37, 293], [290, 1, 39]):
        ok, worst = close(feed(eng, "p", toks, cuts), want, lim)
        assert ok, (cuts, worst)
    got = [eng.replay_step([("g", toks[a:b], [b - a - 1])]) for a, b in ((0, 200), (200, 330))]
    assert eng.runner.graph_replays > 0
    ok, worst = close(torch.cat(got), want[[199, 329]], lim[[199, 329]])
    assert ok, worst


# ------------------------------------------------------------------------------------------- far keys and window edges
def _one_layer(layer, seed=11):
    """The query of token 91 points along the key of token 92: that key's score stands out among hundreds (attention), or
    its share of a slowly decaying state does.  Coordinates 0 and 1 of the embedding belong to the two tokens."""
    cfg = config([layer], vocab=96, width=64)
    w = oracle.random_weights(cfg, seed)
    w["embed"][:, :2] = 0.0
    w["embed"][92, 0] = w["embed"][91, 1] = 8.0
    w["l0.norm1"].fill_(1.0)
    return cfg, w


def _aim(w, p, factor=1.0):
    w[p + "k"][:, 0] *= 2.0
    w[p + "q"][:, 1] = w[p + "k"][:, 0] * factor
    for n in "qkv":
        if p + n + ".conv" in w:
            w[p + n + ".conv"].zero_()
            w[p + n + ".conv"][:, -1] = 1.0


def _window_model(kind, d, dv, window, keep):
    if kind == "attention":
        cfg, w = _one_layer(attention(3, 3, d, dv, (window, keep), rotation(8, base=1e5), 12.0 / d))
        p = "l0.mix."
        w[p + "q.norm"].fill_(1.0)
        w[p + "k.norm"].fill_(1.0)
    else:
        cfg, w = _one_layer(parallel(3, 3, d, dv, (window, keep), rotation(8, base=1e5), 1.0, 3, 30.0, 2, 8, 8, [0.9, 0.99]))
        p = "l0.mix.left."
        w["l0.mix.right.out"].zero_()
        for n in "qkv":
            w[p + n + ".b"] *= 0.2
    _aim(w, p, 24 / d)
    return cfg, w


def _far_model(kind):
    if kind == "latent":
        cfg, w = _one_layer(latent(3, 24, 20, 40, 32, 1.6))
        p = "l0.mix."
        # latents and query latents carry the two coordinates in a dimension of their own
        for n in ("dq", "dkv"):
            w[p + n][:, :2] = 0.0
            w[p + n][0] = 0.0
            w[p + n + ".norm"].fill_(1.0)
        w[p + "dkv"][0, 0] = w[p + "dq"][0, 1] = 4.0
        w[p + "uq"][:, 0] = w[p + "uk"][:, 0]
    else:
        cfg, w = _one_layer(parallel(2, 2, 16, 16, (4, 0), rotation(8), 0.25, 2, 5.0, 3, 24, 20, [0.9999] * 3))
        w["l0.mix.left.out"].zero_()
        p = "l0.mix.right."
        own = torch.arange(3) * 24
        # the far token's key has a channel to itself, and queries ask for nothing else
        w[p + "q"].zero_()
        w[p + "k"][own] = 0.0
        w[p + "k"][own, 0] = 3.0
        w[p + "q"][own, 1] = 3.0
    return cfg, w


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("kind", ["latent", "lightning"])
def test_far_keys(tmp_path, kind, target):
    """The last token asks for one far back: at the first places, on both sides of page borders and of the tiles of the
    kernels, and at a border of the portions.  The far token must show in the answer, whether the query ends a prompt's
    portion or is decoded alone."""
    cfg, w = _far_model(kind)
    eng = make_engine(tmp_path, cfg, w, target)
    n = 300
    base = random_tokens(n, 90, 4)
    lim = LIMIT[target[1]]
    for far in (0, 1, 2, 3, 15, 16, 31, 32, 33, 63, 64, 127, 128, 200, 287, 288, 296):
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
@pytest.mark.parametrize("kind", ["attention", "parallel"])
@pytest.mark.parametrize("window,keep,d,dv", [(1, 0, 24, 24), (2, 3, 24, 20), (16, 16, 64, 64), (17, 20, 128, 128), (70, 5, 24, 20),
                                              (64, 65, 128, 96), (128, 4, 128, 128), (9, 130, 144, 200)])
def test_window_and_first_token_edges(tmp_path, kind, window, keep, d, dv, target):
    """A key just inside the window or the last of the kept ones shows; one just outside and the first one not kept do not,
    in prompts and in decoding."""
    cfg, w = _window_model(kind, d, dv, window, keep)
    eng = make_engine(tmp_path, cfg, w, target)
    n, lim = 150, LIMIT[target[1]]
    base = random_tokens(n, 90, 8)
    base[-1] = 91
    plain = expect(cfg, w, base)[-1:]
    places = {n - 1 - back for back in (window - 2, window - 1, window, window + 1)} | {0, keep - 1, keep, keep + 1}
    for at in sorted(places):
        if at < 0 or at >= n - 1:
            continue
        toks = list(base)
        toks[at] = 92
        want = expect(cfg, w, toks)[-1:]
        if n - 1 - at < window or at < keep:
            assert error(plain, want) > 2 * lim, (at, error(plain, want))
        else:
            assert error(plain, want) < 1e-9
        for cuts in ([n], [n - 1, 1], [n - 2, 2], [37]):
            got = feed(eng, "e", toks, cuts)[-1:]
            assert error(got, want) < lim, (at, cuts, error(got, want))


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
    # three decode in one batch, in another order, one left out
    nxt = {f"b{i}": [(7 * i + 3) % cfg["vocab"]] for i in (3, 0, 2)}
    got = eng.replay_step([(r, t, [0]) for r, t in nxt.items()])
    for j, (r, t) in enumerate(nxt.items()):
        toks = reqs[int(r[1])] + t
        want = expect(cfg, w, toks)
        ok, worst = close(got[j:j + 1], want[-1:], row_limits(cfg, w, toks, want, target[1])[-1:])
        assert ok, worst


@pytest.mark.parametrize("target", TARGETS)
def test_pages_between_the_kept_tokens_and_the_window_return(tmp_path, target):
    """A sequence far longer than the pool lives on the pages of its first tokens and its window."""
    cfg, w = weights_of("windows", seed=2)
    toks = random_tokens(240, cfg["vocab"], 12)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target, num_blocks=10)       # 9 pages of 16: two kept, a window of 34, a portion of 40
    ok, worst = close(feed(eng, "r", toks, [40, 1, 1, 30, 2, 25]), want, row_limits(cfg, w, toks, want, target[1]))
    assert ok, worst
    assert eng.scheduler.num_window_released_blocks > 0 and idle(eng)


# ------------------------------------------------------------------------------------------- scheduler and sampling
GREEDY_TARGETS = TARGETS[:2]                                          # fp32: no near ties between two implementations


def _llm(engine):
    from xllm_b200 import LLM
    llm = LLM.__new__(LLM)
    llm.engine, llm.tokenizer, llm._workers = engine, None, None
    return llm


@pytest.mark.parametrize("target", GREEDY_TARGETS)
@pytest.mark.parametrize("policy,overlap,name", [("prefill_first", False, "odd"), ("decode_first", False, "stateless"),
                                                 ("decode_first", True, "odd")])
def test_greedy_generation(tmp_path, policy, overlap, name, target):
    """LLM.generate through the scheduler: more requests than slots, prompts cut by a small token budget."""
    from xllm_b200 import SamplingParams
    cfg, w = weights_of(name, seed=5)
    prompts = [random_tokens(n, cfg["vocab"], 50 + n) for n in (5, 40, 17, 1, 66, 23)]
    eng = make_engine(tmp_path, cfg, w, target, max_tokens_per_batch=24, policy=policy, enable_schedule_overlap=overlap)
    outs = _llm(eng).generate(prompts, SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))
    w64 = {n: t.double() for n, t in w.items()}
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == oracle.greedy(p, 12, cfg, w64)
    if eng.model.state is not None:
        assert idle(eng)


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
    assert eng.scheduler.num_preemptions > 0 and idle(eng)


@pytest.mark.parametrize("target", GREEDY_TARGETS)
def test_shared_prompts_without_state_use_the_prefix_cache(tmp_path, target):
    """A model without recurrent state keeps finished prompts' pages; a prompt that begins alike reads them."""
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("stateless", seed=5)
    first = random_tokens(50, cfg["vocab"], 3)
    eng = make_engine(tmp_path, cfg, w, target)
    assert eng.model.state is None
    w64 = {n: t.double() for n, t in w.items()}
    for p in (first, first[:40] + random_tokens(15, cfg["vocab"], 4)):
        out = _llm(eng).generate([p], SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))[0]
        assert out.outputs[0].token_ids == oracle.greedy(p, 6, cfg, w64)


@pytest.mark.parametrize("target", TARGETS)
def test_sampling_parallel_samples_and_abort(tmp_path, target):
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("windows")
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
    assert idle(eng)
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
    assert args.model_type == "lukinex" and "lukinex" in supported_models() and args.sliding_window == 0
    only = load_model_args(write_checkpoint(tmp_path / "w", *weights_of("windows")))
    assert only.sliding_window == 34 and only.extra["sliding_window_keep"] == 18
    eng = make_engine(tmp_path, cfg, w, ("cpu", "float32"))
    assert eng.model.kv_layout() == [(1, 1, 26), (2, 2, 64), (2, 1, 64), None, (2, 2, 64)]
    # a tensor the model needs is missing: loading says so
    for gone in ("l1.mix.left.q.b", "l1.mix.left.o.b", "l1.mix.left.k.conv", "l1.mix.right.norm", "l2.mix.k.norm", "l0.mix.dkv",
                 "l3.mix.uk", "l0.mix.dq.norm", "l1.mlp.e4.up", "l0.mlp.shared.down", "l0.mlp.router", "l1.norm2b", "head"):
        w2 = dict(w)
        del w2[gone]
        with pytest.raises(KeyError):
            make_engine(tmp_path / "x", cfg, w2, ("cpu", "float32"))
    for at, change in ((1, {"type": "convolution"}), (0, {"mlp": dict(moe(5, 2, 20, 1.0, 12, 1.0), kind="dense")}),
                       (0, {"mlp": moe(5, 6, 20, 1.0, 12, 1.0)}), (0, {"mlp": moe(5, 2, 20, 0.0, 12, 1.0)}),
                       (3, latent(2, 20, 22, 14, 26, 0.3, source=1)), (3, latent(2, 20, 22, 14, 20, 0.3, source=0)),
                       (2, attention(5, 1, 10, 36, (0, 1), rotation(6), 0.5))):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][at].update(change)
        with pytest.raises(ValueError):
            make_engine(tmp_path / "y", bad, w, ("cpu", "float32"))


def test_kernel_sources_of_the_model():
    from xllm_b200 import _build
    from xllm_b200.models import ModelArgs
    from xllm_b200.models.registry import kernel_sources_of
    names = kernel_sources_of(ModelArgs(model_type="lukinex"))
    assert set(names) <= {s.stem for s in _build.kernel_sources()} and {"mla", "linear_attn", "moe"} <= set(names)
