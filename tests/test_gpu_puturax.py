"""The Puturax decoder in the engine against the plain evaluation (``plain_puturax.py``), in 32-bit (sharp) and in bfloat16:
every mixer alone and mixed, whole prompts, prompts long enough to run in chunks side by side, prompts against token-by-token
decoding, prompts in portions down to two tokens, unequal batches against each request alone, slots, states and pages used again
(poisoned), a far token that a row depends on, long decoding, the first tokens, the stream after every layer, greedy generation
through ``Engine.generate`` / ``generate_many`` (captured graphs and eager), the replay program and the command line as child
processes, configurations drawn at random, sublayers on streams of their own against everything in turn (the same bits)."""

import math

import numpy as np
import pytest
import torch

import puturax_models as M
import plain_puturax as P

pytestmark = pytest.mark.gpu

DTYPES = ["float32", "bfloat16"]
_cache = {}


def model(name, tmp_path_factory):
    if name not in _cache:
        cfg = M.CONFIGS[name]
        tensors = M.draw_weights(cfg, seed=17 + len(name) + ord(name[0]))
        d = M.write_model(cfg, tensors, str(tmp_path_factory.mktemp(f"puturax_{name}")))
        _cache[name] = (cfg, tensors, d, {})
    return _cache[name]


def plain_logits(entry, tokens):
    cfg, tensors, _, memo = entry
    key = tuple(tokens)
    if key not in memo:
        memo[key] = P.forward(cfg, tensors, list(tokens))
    return memo[key]


def engine(entry, dtype, **kw):
    from dryft_b200.engine.api import Engine, EngineOptions

    opts = dict(dtype=dtype, max_batch=8, max_seq_len=512, max_tokens=2048, cuda_graphs=False)
    opts.update(kw)
    return Engine(entry[2], EngineOptions(**opts))


def limits(entry):
    """The bfloat16 limits of this model, from what rounding alone does to a prompt of its own under the plain evaluation."""
    cfg, tensors, _, memo = entry
    if "limits" not in memo:
        memo["limits"] = M.bf16_limits(cfg, tensors, M.prompts(cfg, [120], seed=77)[0])
    return memo["limits"]


def check(entry, got, want, dtype, what):
    M.assert_close(got, want, dtype, what, limits(entry) if dtype != "float32" else None)


def close_all(entry, pairs, dtype, what):
    if dtype == "float32":
        for got, want, label in pairs:
            check(entry, got, want, dtype, f"{what}: {label}")
    else:   # a single bfloat16 row cannot be judged statistically: the rows of all pairs together
        check(entry, torch.cat([g.detach().float().cpu() for g, _, _ in pairs]), torch.cat([w for _, w, _ in pairs]), dtype, what)


def decode_together(eng, slots, batch, heads):
    """Decode the rest of every request of ``batch`` one token a step; requests end (and give back what they hold) one
    after another.  Returns request index -> list of logits rows."""
    live, step = [b for b in range(len(batch)) if heads[b] < len(batch[b])], 0
    eng.cache.close_sequences([slots[b] for b in range(len(batch)) if b not in live])
    rows = {b: [] for b in live}
    while live:
        got = eng.stepper.step([slots[b] for b in live], [[batch[b][heads[b] + step]] for b in live], [[0]] * len(live))
        for r, b in enumerate(live):
            rows[b].append(got[r:r + 1])
        step += 1
        done = [b for b in live if heads[b] + step >= len(batch[b])]
        eng.cache.close_sequences([slots[b] for b in done])
        live = [b for b in live if b not in done]
    return rows


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(M.CONFIGS))
def test_whole_prompts_decoding_portions_and_batches(tmp_path_factory, name, dtype):
    entry = model(name, tmp_path_factory)
    cfg = entry[0]
    eng = engine(entry, dtype)
    reqs = M.prompts(cfg, [1, 2, 23, 65, 131, 200], seed=3)
    with torch.inference_mode():
        # whole prompts, logits at every place (the first tokens included)
        pairs = []
        for toks in reqs:
            s = eng.cache.open_sequences(1)
            got = eng.stepper.step(s, [toks], [list(range(len(toks)))])
            eng.cache.close_sequences(s)
            pairs.append((got, plain_logits(entry, toks), f"prompt of {len(toks)}"))
        close_all(entry, pairs, dtype, f"{name} whole prompts")
        # a short head at once, the rest token by token (page edges pass over decoded tokens)
        for toks, head in ((reqs[3], 1), (reqs[4], 40), (reqs[5], 129)):
            s = eng.cache.open_sequences(1)
            rows = [eng.stepper.step(s, [toks[:head]], [[head - 1]])]
            for t in range(head, len(toks)):
                rows.append(eng.stepper.step(s, [[toks[t]]], [[0]]))
            eng.cache.close_sequences(s)
            check(entry, torch.cat(rows), plain_logits(entry, toks)[head - 1:], dtype, f"{name} decoding {len(toks)} from {head}")
        # portions of several sizes, down to two tokens (a state and a last token handed on)
        for portion in (2, 7, 64, 97):
            toks = reqs[4]
            s = eng.cache.open_sequences(1)
            rows = []
            for c0 in range(0, len(toks), portion):
                piece = toks[c0:c0 + portion]
                rows.append(eng.stepper.step(s, [piece], [list(range(len(piece)))]))
            eng.cache.close_sequences(s)
            check(entry, torch.cat(rows), plain_logits(entry, toks), dtype, f"{name} portions of {portion}")
        # an unequal batch of prompts (one of a single token), then decoded together; shorter requests end earlier
        batch = [reqs[2], reqs[5], reqs[3], reqs[1], reqs[0] + reqs[2]]
        heads = [max(1, len(t) - 12) for t in batch]
        slots = eng.cache.open_sequences(len(batch))
        got = eng.stepper.step(slots, [t[:h] for t, h in zip(batch, heads)], [list(range(h)) for h in heads])
        at, pairs = 0, []
        for t, h in zip(batch, heads):
            pairs.append((got[at:at + h], plain_logits(entry, t)[:h], f"prompt of {h}"))
            at += h
        close_all(entry, pairs, dtype, f"{name} batched prompts")
        rows = decode_together(eng, slots, batch, heads)
        close_all(entry, [(torch.cat(r), plain_logits(entry, batch[b])[heads[b]:], f"request {b}") for b, r in rows.items()],
                  dtype, f"{name} batched decoding")
    eng.cache.check()


@pytest.mark.parametrize("name", ["mixed", "sizes"])
def test_the_stream_after_every_layer(tmp_path_factory, name):
    entry = model(name, tmp_path_factory)
    cfg, tensors = entry[0], entry[1]
    eng = engine(entry, "float32")
    toks = M.prompts(cfg, [90], seed=8)[0]
    want = []
    P.forward(cfg, tensors, toks, lambda i, x: want.append(x.clone()))
    got = []
    eng.model.layer_tap = lambda i, block, res: got.append(res.x.double().cpu())
    with torch.inference_mode():
        s = eng.cache.open_sequences(1)
        eng.stepper.step(s, [toks], [[0]])
        eng.cache.close_sequences(s)
    assert len(got) == len(want) == len(cfg["layers"])
    for i, (g, w) in enumerate(zip(got, want)):
        assert float((g - w).abs().max()) <= 2e-5 * float(w.abs().max()), f"layer {i}"


@pytest.mark.parametrize("dtype", DTYPES)
def test_pages_slots_and_states_used_again_hold_nothing_of_their_last_holder(tmp_path_factory, dtype):
    entry = model("mixed", tmp_path_factory)
    cfg = entry[0]
    # room for little more than one request: every request reuses the slot, the states and the pages of the one before
    eng = engine(entry, dtype, max_batch=1, max_seq_len=256, max_tokens=256)
    reqs = M.prompts(cfg, [150, 90, 201, 33], seed=5)
    with torch.inference_mode():
        for i, toks in enumerate(reqs):
            s = eng.cache.open_sequences(1)
            head = len(toks) - 9
            rows = [eng.stepper.step(s, [toks[:head]], [list(range(head))])]
            for t in range(head, len(toks)):
                rows.append(eng.stepper.step(s, [[toks[t]]], [[0]]))
            eng.cache.close_sequences(s)
            check(entry, torch.cat(rows), plain_logits(entry, toks), dtype, f"request {i} on a reused slot and pages")
            for g in eng.cache._groups:        # what the freed pages hold must never matter again
                g.k.fill_(float("nan"))
                if g.v is not None:
                    g.v.fill_(float("nan"))
            for st in eng.cache._state_tensors():      # ... and neither must a freed slot's states and last tokens
                st.fill_(float("nan"))
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(tmp_path_factory, dtype):
    entry = model("mixed", tmp_path_factory)
    cfg = entry[0]
    eng = engine(entry, dtype, max_batch=2, max_seq_len=512, max_tokens=2048)
    toks = M.prompts(cfg, [330], seed=9)[0]
    with torch.inference_mode():
        s = eng.cache.open_sequences(1)
        rows = [eng.stepper.step(s, [toks[:3]], [[0, 1, 2]])]
        for t in range(3, len(toks)):
            rows.append(eng.stepper.step(s, [[toks[t]]], [[0]]))
        eng.cache.close_sequences(s)
    check(entry, torch.cat(rows), plain_logits(entry, toks), dtype, "330 tokens, nearly all decoded one by one")
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "tc"])
def test_greedy_generation_through_the_entry_point(tmp_path_factory, name, dtype):
    entry = model(name, tmp_path_factory)
    cfg, tensors = entry[0], entry[1]
    eng = engine(entry, dtype, cuda_graphs=True, max_batch=4)
    prompts = M.prompts(cfg, [5, 19, 40], seed=21)
    n_new = 12
    steps = list(eng.generate(prompts, n_new))
    got = [[st[b] for st in steps] for b in range(len(prompts))]
    many = eng.generate_many(prompts + prompts[:2], n_new)
    assert many[:3] == got and many[3:] == got[:2]
    if dtype == "float32":
        for b, p in enumerate(prompts):
            assert got[b] == P.greedy(cfg, tensors, p, n_new), f"request {b}"
    else:
        # bfloat16 may part ways with the plain tokens at a close call, and the contexts differ from then on.  Teacher-forced
        # instead: under the plain model, fed our tokens, each of our tokens is the best one up to what rounding does
        for b, p in enumerate(prompts):
            lg = plain_logits(entry, list(p) + got[b][:-1])[len(p) - 1:]
            ours = lg.gather(1, torch.tensor(got[b])[:, None])[:, 0]
            lost = (lg.max(dim=-1).values - ours) / lg.std(dim=-1)
            assert float(lost.max()) <= 0.3, f"request {b}: token {int(lost.argmax())} loses {float(lost.max()):.3g} spreads to the plain model's best"
    eager = engine(entry, dtype, cuda_graphs=False, max_batch=4)     # graphs and eager steps choose the same tokens
    assert eager.generate_many(prompts, n_new) == got
    if dtype == "float32":
        chunked = engine(entry, dtype, cuda_graphs=False, max_batch=4, prefill_chunk_tokens=16)
        assert chunked.generate_many(prompts, n_new) == got


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_as_a_child_process(tmp_path_factory, tmp_path, dtype):
    import json
    import os
    import subprocess
    import sys

    import helpers as H

    entry = model("mixed", tmp_path_factory)
    cfg = entry[0]
    reqs = M.prompts(cfg, [70, 31, 2], seed=33)
    out = str(tmp_path / "out")
    steps = [{"step": 0, "entries": [{"id": f"r{i}", "tokens": t[:-1] if len(t) > 2 else t[:1], "want": [0, len(t) - 2] if len(t) > 2 else [0]}
                                     for i, t in enumerate(reqs)], "end": []},
             {"step": 1, "entries": [{"id": f"r{i}", "tokens": [t[-1]], "want": [0]} for i, t in enumerate(reqs)], "end": ["r0", "r1", "r2"]},
             {"step": 2, "entries": [{"id": "r0", "tokens": reqs[1], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "r0", "tokens": [5], "want": [0]}], "end": ["r0"]}]
    proc = subprocess.run([sys.executable, os.path.join(H.ROOT, "bin", "trace_run"), "--model", entry[2], "--dtype", dtype,
                           "--out", out, "--max-tokens", "256"], input="".join(json.dumps(s) + "\n" for s in steps),
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-2000:]
    assert [ln for ln in proc.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(4)]
    read = lambda n: torch.from_numpy(np.fromfile(os.path.join(out, f"{n}.f32"), dtype="<f4").reshape(-1, cfg["vocab"]).copy())
    want0 = torch.cat([plain_logits(entry, t)[[0, len(t) - 2] if len(t) > 2 else [0]] for t in reqs])
    check(entry, read(0), want0, dtype, "replayed prompts")
    check(entry, read(1), torch.cat([plain_logits(entry, t)[-1:] for t in reqs]), dtype, "replayed decode step")
    check(entry, read(3), plain_logits(entry, reqs[1] + [5])[-1:], dtype, "a request id used again")


def test_command_line_generates(tmp_path_factory):
    import json
    import subprocess
    import sys

    import helpers as H

    entry = model("mixed", tmp_path_factory)
    cfg, tensors = entry[0], entry[1]
    base = [sys.executable, "-m", "dryft_b200", "generate", "--model", entry[2], "--dtype", "float32", "--max-batch", "4",
            "--max-seq-len", "128", "--prompt-ids", "5,17,3,60,9", "--prompt-ids", "7,7,7", "--max-new-tokens", "6"]
    greedy = subprocess.run(base, capture_output=True, text=True, timeout=600, cwd=H.ROOT)
    assert greedy.returncode == 0, greedy.stderr[-2000:]
    rows = [json.loads(ln) for ln in greedy.stdout.splitlines() if ln.startswith("{")]
    assert [r["tokens"] for r in rows] == [P.greedy(cfg, tensors, p, 6) for p in ([5, 17, 3, 60, 9], [7, 7, 7])]


@pytest.mark.parametrize("dtype", DTYPES)
def test_forty_unequal_requests_at_once(tmp_path_factory, dtype):
    """More rows than the few-row products take; requests end one after another."""
    entry = model("mixed", tmp_path_factory)
    cfg = entry[0]
    eng = engine(entry, dtype, max_batch=64, max_seq_len=256, max_tokens=8192)
    reqs = M.prompts(cfg, [3 + (7 * i) % 50 for i in range(40)], seed=4)
    with torch.inference_mode():
        slots = eng.cache.open_sequences(len(reqs))
        heads = [max(1, len(r) - 5) for r in reqs]
        got = eng.stepper.step(slots, [r[:h] for r, h in zip(reqs, heads)], [[h - 1] for h in heads])
        pairs = [(got[i:i + 1], plain_logits(entry, reqs[i])[heads[i] - 1:heads[i]], f"prompt {i}") for i in range(len(reqs))]
        rows = decode_together(eng, slots, reqs, heads)
        pairs += [(torch.cat(r), plain_logits(entry, reqs[b])[heads[b]:], f"request {b}") for b, r in rows.items() if r]
    close_all(entry, pairs, dtype, "forty requests")
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_sublayers_on_streams_of_their_own_give_the_same_bits(tmp_path_factory, dtype):
    """Few-row steps run the feed-forward beside the mixer, and the two mixers of a pair beside each other, on side streams
    (parallel branches of a captured step): the logits are the same bits as with everything in turn, eagerly and replayed."""
    entry = model("mixed", tmp_path_factory)
    cfg = entry[0]
    reqs = M.prompts(cfg, [70, 31, 2, 9], seed=14)
    rows = {}
    for branch in (16, 0):
        eng = engine(entry, dtype, branch_rows=branch)
        with torch.inference_mode():
            slots = eng.cache.open_sequences(len(reqs))
            got = [eng.stepper.step(slots, reqs, [[len(t) - 1] for t in reqs])]     # four rows wanted of a step of many
            for t in range(20):
                got.append(eng.stepper.step(slots, [[(7 * t + b) % cfg["vocab"]] for b in range(len(reqs))], [[0]] * len(reqs)))
            eng.cache.close_sequences(slots)
            torch.cuda.synchronize()
        rows[branch] = torch.cat(got).cpu()
        toks = engine(entry, dtype, branch_rows=branch, cuda_graphs=True, max_batch=4).generate_many(reqs, 10)
        rows[("tokens", branch)] = toks
    assert torch.equal(rows[16], rows[0])
    assert rows[("tokens", 16)] == rows[("tokens", 0)]
    want = torch.cat([plain_logits(entry, t)[-1:] for t in reqs])
    check(entry, rows[16][:len(reqs)], want, dtype, "prompts before the branched steps")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "sizes", "tc"])
def test_prompts_long_enough_to_run_in_chunks(tmp_path_factory, name, dtype):
    """Steps of 256 tokens and more cut the recurrence into chunks: whole, in pieces of unequal lengths, and batched."""
    entry = model(name, tmp_path_factory)
    cfg = entry[0]
    eng = engine(entry, dtype)
    a, b, c = M.prompts(cfg, [330, 270, 41], seed=6)
    with torch.inference_mode():
        s = eng.cache.open_sequences(1)
        rows = [eng.stepper.step(s, [a[p0:p1]], [list(range(p1 - p0))]) for p0, p1 in ((0, 40), (40, 310), (310, 330))]
        eng.cache.close_sequences(s)
        check(entry, torch.cat(rows), plain_logits(entry, a), dtype, f"{name} in pieces around a long one")
        slots = eng.cache.open_sequences(3)
        got = eng.stepper.step(slots, [a[:-1], c[:-1], b[:-1]], [list(range(len(t) - 1)) for t in (a, c, b)])
        more = eng.stepper.step(slots, [a[-1:], c[-1:], b[-1:]], [[0]] * 3)
        eng.cache.close_sequences(slots)
        check(entry, got, torch.cat([plain_logits(entry, t)[:-1] for t in (a, c, b)]), dtype, f"{name} long prompts in a batch")
        check(entry, more, torch.cat([plain_logits(entry, t)[-1:] for t in (a, c, b)]), dtype, f"{name} decoding behind them")
    eng.cache.check()


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_far_token_that_a_row_depends_on(tmp_path_factory, dtype):
    """The recurrence decays at once and the bias is weak, so that only attention reaches far; the last token asks for the first
    one's key, which stands out.  Changing that token must move the row, in a prompt and in decoding, as the plain model says."""
    cfg = M.config([M.pair(heads=2, kv_heads=1, dim=16, vdim=16, softcap=30.0, q_temp=(0.2, 100), scale=1.5, right_scale=0.2, mlp=None)], width=32, vocab=64)
    tensors = M.draw_weights(cfg, seed=3)
    tensors["l0.mix.right.w0"].fill_(4.0)
    tensors["l0.mix.left.r1"].fill_(0.25)
    toks = M.prompts(cfg, [260], seed=2)[0]
    x = P.layer_norm1(tensors["embed"].double() * 3.0, tensors["l0.norm1"].double(), 1e-5)
    q, k = tensors["l0.mix.left.q"].double(), tensors["l0.mix.left.k"].double()
    # the key of token 9 points where the query of token 5 looks
    qv = (q @ x[5]).view(2, 16).mean(0)
    kx = x[9] / (x[9] * x[9]).sum()
    tensors["l0.mix.left.k"] = (k + torch.outer(4.0 * qv / qv.norm() * math.sqrt(16) - k @ x[9], kx)).to(torch.bfloat16)
    toks = [t if t not in (5, 9) else 11 for t in toks]
    toks[0], toks[-1] = 9, 5
    d = M.write_model(cfg, tensors, str(tmp_path_factory.mktemp("puturax_far")))
    entry = (cfg, tensors, d, {})
    other = [12] + toks[1:]
    w0, w1 = plain_logits(entry, toks)[-1:], plain_logits(entry, other)[-1:]
    assert float(M.row_errors(w1, w0)) > 0.2                 # the far token carries the row
    eng = engine(entry, dtype)
    with torch.inference_mode():
        for t, want in ((toks, w0), (other, w1)):
            for head in (len(t), len(t) - 1, 3):
                s = eng.cache.open_sequences(1)
                got = eng.stepper.step(s, [t[:head]], [[head - 1]])
                for j in range(head, len(t)):
                    got = eng.stepper.step(s, [[t[j]]], [[0]])
                eng.cache.close_sequences(s)
                assert float(M.row_errors(got, want)) <= (M.FP32_TOL if dtype == "float32" else 0.03), f"{head} tokens at once"


def _random_config(seed):
    """A configuration drawn at random: layer kinds and order, every size, every constant."""
    import random

    r = random.Random(seed)
    layers = []
    for i in range(r.randint(2, 4)):
        kind = r.choice(["dense", "moe", "moe", None])
        if kind == "dense":
            kind = {"kind": "dense", "ff": r.randint(5, 70)}
        elif kind == "moe":
            count = r.randint(1, 4)
            each = r.randint(1, 4)
            keep = r.randint(1, count)
            kind = M.moe(r.randint(4, 40), count * each, r.randint(1, keep * each), r.choice([(count, keep), (count, keep), None]), r.choice([None, r.randint(4, 40)]))
        if r.random() < 0.35:
            layers.append(M.latent(r.randint(1, 5), r.randint(2, 40), 2 * r.randint(0, 9), r.randint(2, 40), r.randint(3, 50), r.randint(3, 90),
                                   r.choice([37.0, 1000.0, 250000.0]), mlp=kind))
            continue
        kv = r.randint(1, 3)
        layers.append(M.pair(kv * r.randint(1, 4), kv, r.randint(2, 48), r.randint(2, 48), r.choice([None, round(r.uniform(2.0, 30.0), 2)]),
                             r.choice([None, (round(r.uniform(0.05, 1.0), 2), r.choice([1, 3, 17, 64, 500]))]), None, r.randint(1, 4), r.randint(2, 80),
                             r.choice([None, round(r.uniform(0.3, 2.0), 2)]), r.choice([None, round(r.uniform(0.3, 2.0), 2)]), mlp=kind))
    return M.config(layers, width=r.choice([24, 36, 50, 52, 64]), vocab=r.randint(40, 300), eps=r.choice([1e-6, 1e-5, 3e-4]),
                    emb_scale=r.choice([None, round(r.uniform(0.3, 12.0), 2)]))


@pytest.mark.parametrize("seed", range(10))
def test_configurations_drawn_at_random(tmp_path, seed):
    cfg = _random_config(seed)
    tensors = M.draw_weights(cfg, seed=100 + seed)
    entry = (cfg, tensors, M.write_model(cfg, tensors, str(tmp_path / "m")), {})
    reqs = M.prompts(cfg, [170, 1, 33], seed=seed)
    for dtype in DTYPES:
        eng = engine(entry, dtype, max_batch=4, max_seq_len=256, max_tokens=1024)
        with torch.inference_mode():
            heads = [max(1, len(t) - 6) for t in reqs]
            slots = eng.cache.open_sequences(len(reqs))
            got = eng.stepper.step(slots, [t[:h] for t, h in zip(reqs, heads)], [list(range(h)) for h in heads])
            at, pairs, spans = 0, [], [(t, 0, h) for t, h in zip(reqs, heads)]
            for t, h in zip(reqs, heads):
                pairs.append((got[at:at + h], plain_logits(entry, t)[:h], f"prompt of {h}"))
                at += h
            rows = decode_together(eng, slots, reqs, heads)
            pairs += [(torch.cat(v), plain_logits(entry, reqs[b])[heads[b]:], f"request {b} decoded") for b, v in rows.items() if v]
            spans += [(reqs[b], heads[b], len(reqs[b])) for b, v in rows.items() if v]
        what = f"random configuration {seed} ({[l['type'] for l in cfg['layers']]})"
        if dtype == "float32":
            # a drawn model may have rows that 32-bit arithmetic cannot hold (a choice or a norm that cancels): the plain evaluation in
            # 32-bit shows it; its worst row bounds ours, and the typical row stays sharp
            for (got_, want_, label), (t, a, b) in zip(pairs, spans):
                own = M.row_errors(P.forward(cfg, tensors, t, number=torch.float32), plain_logits(entry, t)).double().cpu()
                e = M.row_errors(got_, want_).double().cpu()
                assert torch.isfinite(got_).all() and float(e.median()) <= M.FP32_TOL and float(e.max()) <= max(M.FP32_TOL, 2.0 * float(own.max())), \
                    f"{what}: {label} off by {float(e.max()):.3g}"
        else:
            # heads of two or three values and widths of 24 make bfloat16 rounding large in some of these models: the sharp
            # comparison is the 32-bit one; here the typical row must be close and every row finite
            got_all = torch.cat([g.detach().float().cpu() for g, _, _ in pairs])
            assert torch.isfinite(got_all).all(), what
            e = M.row_errors(got_all, torch.cat([w for _, w, _ in pairs]))
            limit = M.bf16_limits(cfg, tensors, reqs[0])[0]      # what rounding alone does to the very prompt that is tested
            assert float(e.median()) <= limit, f"{what}: median row off by {float(e.median()):.3g} (limit {limit:.3g})"
        eng.cache.check()
