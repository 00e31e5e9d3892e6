"""Femirax through the engine (loading, cache, state slots, scheduler, sampling) against a plain implementation of its
equations: whole prompts, portions, token by token, mixed batches, reused pages and slots, far keys, greedy generation."""
import io
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import femirax_oracle as oracle
from femirax_common import (CONFIGS, LIMIT, TARGETS, config, error, expect, feed, make_engine, parallel, random_tokens,
                            retention, weights_of, write_checkpoint)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


@pytest.mark.parametrize("target", TARGETS)
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_portions_and_decoding_match_the_whole_prompt(tmp_path, name, target):
    cfg, w = weights_of(name)
    toks = random_tokens(75, cfg["vocab"], 1)
    want = expect(cfg, w, toks)
    eng = make_engine(tmp_path, cfg, w, target)
    lim = LIMIT[target[1]]
    for cuts in ([75], [2, 3, 17], [16], [40, 1, 1, 1], [1], [33, 2, 15, 16, 5]):
        assert error(feed(eng, "r", toks, cuts), want) < lim, (name, cuts)
    assert len(eng.model.state.free) == 4 and eng.scheduler.block_stats(0).num_used == 0


@pytest.mark.parametrize("target", TARGETS)
def test_layer_streams(tmp_path, target):
    """The residual stream behind every layer of one short prompt."""
    cfg, w = weights_of("odd")
    toks = random_tokens(21, cfg["vocab"], 2)
    want = []
    oracle.forward(toks, cfg, {n: t.double() for n, t in w.items()}, want)
    eng = make_engine(tmp_path, cfg, w, target)
    from xllm_b200.models import femirax
    got, plain = [], femirax.residual_update

    def spy(x, y, w=None, **kw):
        r = plain(x, y, w=w, **kw)
        if w is not None and kw.get("y2") is None:                   # the side input joins: end of a layer
            got.append(r[0].double().cpu().clone())
        return r

    femirax.residual_update = spy
    try:
        from xllm_b200.api.embedding import hidden_states
        hidden_states(eng, toks)
    finally:
        femirax.residual_update = plain
    assert len(got) == len(want)
    for g, e in zip(got, want):
        assert float((g - e).pow(2).mean().sqrt() / e.pow(2).mean().sqrt()) < (1e-5 if target[1] == "float32" else 0.02)


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
            n = int(rng.choice([1, 1, 2, 3, 16, 29]))
            n = min(n, len(reqs[r]) - at)
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
            assert error(torch.stack([x for _, x in rows]), want[r][at]) < LIMIT[target[1]], r
    assert steps > 10 and len(eng.model.state.free) == 4 and eng.scheduler.block_stats(0).num_used == 0
