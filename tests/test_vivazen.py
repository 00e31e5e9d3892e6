"""Vivazen through the engine (loading, cache, state slots, scheduler, sampling) against a plain implementation of its equations:
whole prompts, portions, token by token, mixed batches, reused pages and slots, far keys, window edges, sinks, greedy generation."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

import vivazen_oracle as oracle
from femirax_common import LIMIT, TARGETS, close, error, feed, make_engine, random_tokens, write_checkpoint
from vivazen_common import CONFIGS, again, attention, config, expect, latent, rotation, row_limits, weights_of

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
    """The residual stream behind every layer of one short prompt, lent tensors included."""
    cfg, w = weights_of(name)
    toks = random_tokens(21, cfg["vocab"], 2)
    want = []
    oracle.forward(toks, cfg, {n: t.double() for n, t in w.items()}, want)
    eng = make_engine(tmp_path, cfg, w, target)
    from xllm_b200.models import vivazen
    got, plain = [], vivazen.VivazenLayer.forward

    def spy(self, x, *a):
        h = plain(self, x, *a)
        got.append(x.double().cpu().clone())
        return h

    vivazen.VivazenLayer.__call__ = spy
    try:
        from xllm_b200.api.embedding import hidden_states
        hidden_states(eng, toks)
    finally:
        vivazen.VivazenLayer.__call__ = plain
    assert len(got) == len(want)
    for g, e in zip(got, want):
        assert float((g - e).pow(2).mean().sqrt() / e.pow(2).mean().sqrt()) < (1e-5 if target[1] == "float32" else 0.03)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", ["odd", "aligned", "wide", "windows"])
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
@pytest.mark.parametrize("graph", [False, True])
def test_long_prompts_expand_their_latents(tmp_path, graph):
    """Prompts of hundreds of tokens through keys and values made from the latents, whole, behind an earlier portion and beside
    decoding requests, eager and captured."""
    cfg, w = weights_of("aligned", seed=4)
    toks = random_tokens(330, cfg["vocab"], 2)
    want = expect(cfg, w, toks)
    lim = row_limits(cfg, w, toks, want, "bfloat16")
    eng = make_engine(tmp_path, cfg, w, ("cuda:0", "bfloat16"), enable_graph=graph)
    from xllm_b200 import ops
    calls, plain = [], ops.ragged_prefill_attention
    ops.ragged_prefill_attention = lambda *a, **k: (calls.append(1), plain(*a, **k))[1]
    try:
        for cuts in ([330], [37, 293], [290, 1, 39]):
            ok, worst = close(feed(eng, "p", toks, cuts), want, lim)
            assert ok, (cuts, worst)
        assert len(calls) >= 6                                        # two layers have rows wide enough
        short = random_tokens(20, cfg["vocab"], 3)
        eng.replay_step([("d", short[:19], [])])
        both = eng.replay_step([("d", short[19:], [0]), ("p", toks[:300], [0, 150, 299]), ("q", toks[:9], [8])])
        last = eng.replay_step([("d", [5], []), ("p", toks[300:], [29])])
    finally:
        ops.ragged_prefill_attention = plain
    ws = expect(cfg, w, short)
    assert close(both[:1], ws[-1:], row_limits(cfg, w, short, ws, "bfloat16")[-1:])[0]
    at = [0, 150, 299, 8]
    assert close(both[1:], want[at], lim[at])[0] and close(last, want[-1:], lim[-1:])[0]
    assert (eng.runner.graph_replays > 0) == graph


# ------------------------------------------------------------------------------------------- far keys and window edges
def _one_layer(layer, seed=11, groups=1):
    """The query of token 91 points along the key of token 92: that key's score stands out among hundreds.  Coordinates 0 and 1 of the
    embedding belong to the two tokens."""
    cfg = config([layer], vocab=96, width=64, groups=groups, alpha=0.5)
    w = oracle.random_weights(cfg, seed)
    w["embed"][:, :2] = 0.0
    w["embed"][92, 0] = w["embed"][91, 1] = 8.0
    return cfg, w


def _talking_model(heads, kv, d, dv):
    cfg, w = _one_layer(attention(heads, kv, d, dv, 3, 1.2, 30.0))
    p = "l0.mix."
    for n in "qkv":
        w[p + n + ".conv"].zero_()
        w[p + n + ".conv"][:, -1] = 1.0
    for n in "qk":
        w[p + n + ".norm"].fill_(1.0)
    w[p + "k"][:, 0] *= 2.0
    w[p + "q"][:, 1] = w[p + "k"].view(kv, d, -1)[:, None, :, 0].expand(kv, heads // kv, d).reshape(-1)
    return cfg, w


def _window_model(heads, d, dv, rank, rot, window):
    cfg, w = _one_layer(latent(heads, d, dv, rank, rotation(rot, base=1e5), window, 1.0))
    p = "l0.mix."
    # latents carry the far token's coordinate in a dimension of their own, which a query asks for
    w[p + "dkv"][:, :2] = 0.0
    w[p + "dkv"][0] = 0.0
    w[p + "dkv"][0, 0] = 4.0
    w[p + "dkv.norm"].fill_(1.0)
    w[p + "uk"][:, 0] = 1.0
    w[p + "q"].view(heads, d + rot, -1)[:, :d, 1] = 6.0 / d
    w[p + "g"][:, 1] = 0.5
    return cfg, w


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("sizes", [(4, 2, 24, 20), (16, 4, 128, 128)])
def test_far_keys(tmp_path, sizes, target):
    """The last token asks for one far back: at the first places, on both sides of page borders and of the tiles of the kernels, and
    at a border of the portions.  The far token must show in the answer, whether the query ends a prompt's portion or is decoded
    alone."""
    cfg, w = _talking_model(*sizes)
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
        assert seen > 2 * lim, (far, seen)                           # leaving the far key out would show
        for cuts in ([n], [64, 33, 2, 200, 1], [n - 3, 3], [n - 2, 2], [n - 1, 1]):
            at, i = 0, 0
            while at < n:
                m = min(cuts[i % len(cuts)], n - at)
                got = eng.replay_step([("f", toks[at:at + m], [m - 1] if at + m == n else [])])
                at, i = at + m, i + 1
            eng.replay_end("f")
            assert error(got, want) < lim, (far, cuts)


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("heads,d,dv,rank,rot,window", [(3, 24, 20, 40, 8, 1), (3, 24, 20, 40, 8, 2), (2, 32, 32, 88, 32, 16),
                                                        (4, 64, 128, 200, 32, 17), (2, 64, 64, 448, 64, 64), (2, 40, 24, 512, 64, 70),
                                                        (2, 64, 128, 512, 64, 128)])
def test_window_edges(tmp_path, heads, d, dv, rank, rot, window, target):
    """A key just inside the window shows; one just outside does not, in prompts and in decoding."""
    cfg, w = _window_model(heads, d, dv, rank, rot, window)
    eng = make_engine(tmp_path, cfg, w, target)
    n, lim = 150, LIMIT[target[1]]
    base = random_tokens(n, 90, 8)
    base[-1] = 91
    plain = expect(cfg, w, base)[-1:]
    for back in (window - 2, window - 1, window, window + 1):
        at = n - 1 - back
        if at < 0 or at >= n - 1:
            continue
        toks = list(base)
        toks[at] = 92
        want = expect(cfg, w, toks)[-1:]
        if back < window:
            assert error(plain, want) > 2 * lim, (at, error(plain, want))
        else:
            assert error(plain, want) < 1e-9
        for cuts in ([n], [n - 1, 1], [n - 2, 2], [37]):
            got = feed(eng, "e", toks, cuts)[-1:]
            assert error(got, want) < lim, (at, cuts, error(got, want))


@pytest.mark.gpu
def test_window_edges_of_long_portions(tmp_path):
    """Expanded latents: the window's edge of rows in the middle of a portion of hundreds, its context gathered from the edge on."""
    n, window = 500, 100
    cfg, w = _window_model(2, 64, 128, 512, 64, window)
    eng = make_engine(tmp_path, cfg, w, ("cuda:0", "bfloat16"))
    lim = LIMIT["bfloat16"]
    for ask in (140, 227, 228, 356, 499):
        for back in (window - 1, window):
            toks = random_tokens(n, 90, 8)
            toks[ask], toks[ask - back] = 91, 92
            want = expect(cfg, w, toks)[ask:ask + 1]
            for cuts in ([n], [30, 470], [130, 370]):
                assert error(feed(eng, "e", toks, cuts)[ask:ask + 1], want) < lim, (ask, back, cuts)


@pytest.mark.parametrize("target", TARGETS)
def test_sinks_and_scaled_rotation_show(tmp_path, target):
    """Answers with the sinks left out, or with the frequencies unscaled, would differ by more than the limit."""
    cfg = config([latent(4, 32, 24, 80, rotation(32, base=5e3, factor=8.0, original=128), 90, 0.25)], vocab=96, width=64)
    w = oracle.random_weights(cfg, 3)
    w["l0.mix.sink"] += 4.0
    toks = random_tokens(120, 96, 1)
    want = expect(cfg, w, toks)
    off = dict(w, **{"l0.mix.sink": torch.full((4,), -60.0)})
    flat = json.loads(json.dumps(cfg))
    flat["layers"][0]["mixer"]["rot"]["scaling"]["factor"] = 1.0
    assert error(expect(cfg, off, toks), want) > 2 * LIMIT[target[1]] and error(expect(flat, w, toks), want) > 2 * LIMIT[target[1]]
    eng = make_engine(tmp_path, cfg, w, target)
    lim = row_limits(cfg, w, toks, want, target[1])
    for cuts in ([120], [100, 1, 1, 9]):
        ok, worst = close(feed(eng, "s", toks, cuts), want, lim)
        assert ok, (cuts, worst)


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
@pytest.mark.parametrize("name", ["odd", "aligned"])
def test_long_decoding(tmp_path, name, target):
    """A short prompt, then hundreds of tokens one at a time across many page borders and windows."""
    cfg, w = weights_of(name, seed=6)
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
def test_pages_behind_the_windows_return(tmp_path, target):
    """A sequence far longer than the pool lives on the pages of its widest window."""
    cfg, w = weights_of("windows", seed=2)
    toks = random_tokens(240, cfg["vocab"], 12)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target, num_blocks=8)        # 7 pages of 16: a window of 34 and a portion of 40
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
@pytest.mark.parametrize("policy,overlap,name", [("prefill_first", False, "odd"), ("decode_first", False, "windows"),
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


@pytest.mark.gpu
def test_greedy_generation_on_the_tensor_cores(tmp_path):
    """bfloat16 through the scheduler and captured steps: every token is one that the plain implementation finds (nearly) as likely
    as its own."""
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("aligned", seed=5)
    prompts = [random_tokens(n, cfg["vocab"], 50 + n) for n in (5, 140, 17, 1, 66, 23)]
    eng = make_engine(tmp_path, cfg, w, ("cuda:0", "bfloat16"), max_tokens_per_batch=64)
    outs = _llm(eng).generate(prompts, SamplingParams(max_tokens=12, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        toks = p + list(o.outputs[0].token_ids)
        z = expect(cfg, w, toks)[len(p) - 1:-1]
        chosen = z.gather(1, torch.tensor(toks[len(p):])[:, None])[:, 0]
        assert float((z.max(1).values - chosen).max()) < 0.3 * float(z.std())
    assert eng.runner.graph_replays > 0


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


@pytest.mark.parametrize("target", TARGETS)
def test_sampling_parallel_samples_and_abort(tmp_path, target):
    from xllm_b200 import SamplingParams
    cfg, w = weights_of("odd")
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
    assert args.model_type == "vivazen" and "vivazen" in supported_models() and args.sliding_window == 0
    assert load_model_args(write_checkpoint(tmp_path / "w", *weights_of("windows"))).sliding_window == 34
    eng = make_engine(tmp_path, cfg, w, ("cpu", "float32"))
    m = eng.model
    assert m.kv_layout() == [(1, 1, 36), (2, 2, 20), (1, 1, 36), (1, 1, 9), (2, 2, 20), (2, 1, 36)]
    assert m.layers[0] is m.layers[2] and m.layers[1] is m.layers[4] and set(m.state.layers) == {1, 4, 5}
    assert make_engine(tmp_path / "w", *weights_of("windows"), ("cpu", "float32")).model.state is None
    # a tensor the model needs is missing: loading says so
    for gone in ("l0.mix.sink", "l0.mix.g", "l0.mix.uk", "l0.mix.dkv.norm", "l0.norm2", "l1.mix.talk", "l1.mix.k.conv", "l1.mix.q.norm",
                 "l1.mix.o", "l1.mlp.up", "l3.norm1", "final.norm", "head"):
        w2 = dict(w)
        del w2[gone]
        with pytest.raises(KeyError):
            make_engine(tmp_path / "x", cfg, w2, ("cpu", "float32"))
    for at, change in ((1, {"type": "convolution"}), (0, {"mlp": {"ff": 36, "kind": "moe"}}), (3, latent(3, 9, 5, 7, rotation(2), 0, 0.5)),
                       (5, attention(4, 3, 10, 36, 2, 0.4, 30.0)), (5, attention(4, 1, 10, 36, 0, 0.4, 30.0)),
                       (2, again(CONFIGS["odd"]["layers"][3], 0)), (2, {"weights_of": 9}), (0, {"weights_of": 0})):
        bad = json.loads(json.dumps(cfg))
        bad["layers"][at].update(change)
        with pytest.raises(ValueError):
            make_engine(tmp_path / "y", bad, w, ("cpu", "float32"))
    with pytest.raises(ValueError):
        make_engine(tmp_path / "z", dict(cfg, norm={"eps": 1e-5, "groups": 5}), w, ("cpu", "float32"))


def test_kernel_sources_of_the_model():
    from xllm_b200 import _build
    from xllm_b200.models import ModelArgs
    from xllm_b200.models.registry import kernel_sources_of
    names = kernel_sources_of(ModelArgs(model_type="vivazen"))
    assert set(names) <= {s.stem for s in _build.kernel_sources()} and {"mla", "attn_generic", "rope_norm_kv"} <= set(names)
