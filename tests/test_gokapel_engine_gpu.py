"""Gokapel through the engine against the plain implementation: whole prompts, token-by-token decoding from a prompt
and from the very first token, prompts in portions, unequal batches against each request alone, slots, pages and
states used again, decoding far past every chunk, keys at the chunks' edges, a layer run twice with one set of tensors,
generation through the entry points and trace replay (GPU)."""
import copy
import json
import os
import subprocess
import sys

import pytest
import torch

import plain_gokapel as pg
from gokapel_cases import CASES, Want, both, check_rows, dense, delta, folder, make_weights, model, oracle, tokens

pytestmark = pytest.mark.gpu
ROOT = os.path.join(os.path.dirname(os.path.abspath(__file__)), "..")
# max |difference| relative to the oracle's largest logit; in bfloat16 three times a row's own rounding noise on top
TOL = {"float32": 1e-4, "bfloat16": 1.5e-2}
ALL = [(n, d) for n in sorted(CASES) for d in ("float32", "bfloat16")]


@pytest.fixture(scope="module")
def tmp_root(tmp_path_factory):
    return tmp_path_factory.mktemp("gokapel")


def _engine(path, dtype, **kw):
    from tq_kv_b200.engine import Engine
    kw.setdefault("max_tokens", 1024)
    return Engine.from_folder(path, dtype=dtype, **kw)


def _check(got, want, dtype, what):
    check_rows(got, want, dtype, "gokapel " + what, TOL[dtype])


@pytest.mark.parametrize("name,dtype", ALL)
def test_whole_prompts_and_decoding_token_by_token(tmp_root, name, dtype):
    from tq_kv_b200.engine import StepRow
    path = folder(tmp_root, name)
    eng = _engine(path, dtype)
    V = CASES[name]["vocab"]
    for n in (1, 2, 3, 70, 260):                             # the first tokens alone; over one and four pages
        toks = tokens(n, V, 10 + n)
        s = eng.new_sequence()
        _check(eng.step([StepRow(s, toks, list(range(n)))]), oracle(path, toks), dtype, f"{name} whole {n}")
        eng.release(s)
    toks = tokens(260, V, 210)
    want = oracle(path, toks)
    s = eng.new_sequence()
    got = [eng.step([StepRow(s, toks[:150], [149])])]
    for t in range(150, 260):                                # replayed graphs from the second step on
        got.append(eng.step([StepRow(s, [toks[t]], [0])]))
    _check(torch.cat(got), want[149:], dtype, f"{name} decode")
    eng.release(s)
    s = eng.new_sequence()                                   # the same slot, its state zeroed: from the very first token
    got = [eng.step([StepRow(s, [toks[t]], [0])]) for t in range(12)]
    _check(torch.cat(got), want[:12], dtype, f"{name} decode from the first token")
    eng.release(s)
    assert eng.cache.free_slots == eng.cache.max_slots
    eng.cache.book.check()


@pytest.mark.parametrize("name,dtype", ALL)
def test_prompts_in_portions(tmp_root, name, dtype):
    """Portions down to one and two tokens, across page and chunk edges; both memories and the convolution's last
    inputs are handed from portion to portion."""
    from tq_kv_b200.engine import StepRow
    path = folder(tmp_root, name)
    eng = _engine(path, dtype)
    toks = tokens(180, CASES[name]["vocab"], 77)
    want = oracle(path, toks)
    for cuts in ((2, 2, 60, 1, 63, 52), (64, 64, 52), (1, 1, 1, 2, 64, 64, 47), (127, 2, 51), (3, 61, 64, 52)):
        assert sum(cuts) == 180
        s, at, got = eng.new_sequence(), 0, []
        for n in cuts:
            got.append(eng.step([StepRow(s, toks[at:at + n], list(range(n)))]))
            at += n
        _check(torch.cat(got), want, dtype, f"{name} portions {cuts}")
        eng.release(s)


@pytest.mark.parametrize("name,dtype", ALL)
def test_unequal_batches_against_each_alone_and_slots_used_again(tmp_root, name, dtype):
    from tq_kv_b200.engine import StepRow
    path = folder(tmp_root, name)
    eng = _engine(path, dtype, max_tokens=896, max_slots=4)
    V = CASES[name]["vocab"]
    for round_ in range(3):                                  # the same slots, pages and states serve three batches
        lens = [(1, 130, 66), (64, 2, 200), (129, 65, 1)][round_]
        extra = [12, 30, 20]                                 # tokens decoded after the prompt; rows end at different steps
        reqs = [tokens(n + m, V, 100 * round_ + n) for n, m in zip(lens, extra)]
        wants = [oracle(path, r) for r in reqs]
        slots = [eng.new_sequence() for _ in reqs]
        got = [[] for _ in reqs]
        out = eng.step([StepRow(s, r[:n], [n - 1]) for s, r, n in zip(slots, reqs, lens)])
        for i in range(3):
            got[i].append(out[i:i + 1])
        live = [0, 1, 2]
        for step in range(max(extra)):
            live = [i for i in live if step < extra[i]]
            out = eng.step([StepRow(slots[i], [reqs[i][lens[i] + step]], [0]) for i in live])
            for j, i in enumerate(live):
                got[i].append(out[j:j + 1])
            for i in list(live):
                if step + 1 == extra[i]:
                    eng.release(slots[i])                    # its slot, pages and state go back while the others go on
        for i in range(3):
            _check(torch.cat(got[i]), wants[i][lens[i] - 1:], dtype, f"{name} batch round {round_} row {i}")
        assert eng.cache.free_slots == 4
        eng.cache.book.check()


@pytest.mark.parametrize("name,dtype", [x for x in ALL if x[0] != "c"])
def test_a_new_prompt_beside_decoding_rows_and_a_long_decode(tmp_root, name, dtype):
    """A prompt joins a row that decodes (through the paged path), and 400 tokens are decoded one by one: every
    chunk is left and every ring wraps."""
    from tq_kv_b200.engine import StepRow
    path = folder(tmp_root, name)
    eng = _engine(path, dtype)
    V = CASES[name]["vocab"]
    a, b = tokens(440, V, 41), tokens(50, V, 42)
    wa, wb = oracle(path, a), oracle(path, b)
    sa = eng.new_sequence()
    got_a = [eng.step([StepRow(sa, a[:40], [39])])]
    sb = eng.new_sequence()
    out = eng.step([StepRow(sa, [a[40]], [0]), StepRow(sb, b[:50], [0, 49])])      # a prompt beside a decoding row
    got_a.append(out[:1])
    _check(out[1:], Want.cat([wb[0], wb[49]]), dtype, f"{name} the prompt beside a decoding row")
    eng.release(sb)
    for t in range(41, 440):
        got_a.append(eng.step([StepRow(sa, [a[t]], [0])]))
    _check(torch.cat(got_a), wa[39:], dtype, f"{name} long decode")
    eng.release(sa)


# ---- keys at the chunks' edges -----------------------------------------------------------------------------------
def _chunk_cfg():
    """Attention in chunks of 64, 65 and 70 positions with little beside it: few keys carry a row, so that the key that
    enters a chunk or stays outside moves it."""
    return model(120, 64, 1e-5, 2, 1.0, 1.0, [
        {**both(2, 1, 32, 32, 70, 1.0, 16, 1.5, 0.1), "mlp": None},
        {**both(2, 1, 32, 32, 64, 1.0, 16, 1.5, 0.1), "mlp": None},
        {**both(2, 2, 64, 64, 65, 0.5, 16, 1.5, 0.1), "mlp": None},
    ])


def _edge_rows(T):
    """The positions whose keys change when a chunk of 64, 65 or 70 is one longer or shorter: around every edge."""
    return sorted({p for c in (64, 65, 70) for k in range(c, T, c) for p in range(k - 3, k + 4) if 0 <= p < T})


def test_a_chunk_one_position_off_moves_the_rows_at_its_edges():
    """The oracle itself: with any chunk one position longer or shorter, rows that the edge tests read move by a tenth
    of the largest logit or more, many times what float32 and bfloat16 bounds allow."""
    cfg = _chunk_cfg()
    w = make_weights(cfg, 9, sharp=True)
    toks = tokens(200, cfg["vocab"], 13)
    base = pg.decoder(cfg, w, toks)
    scale = float(base.abs().max())
    rows = _edge_rows(200)
    for off in (-1, 1):
        for layer in range(3):
            c2 = copy.deepcopy(cfg)
            c2["layers"][layer]["mixer"]["left"]["mask"]["size"] += off
            moved = float((pg.decoder(c2, w, toks)[rows] - base[rows]).abs().max()) / scale
            assert moved > 0.1, (layer, off, moved)
    noise = (pg.decoder(cfg, w, toks, rounding=lambda t: t.to(torch.bfloat16).to(t.dtype)) - base).abs().amax(dim=1) / scale
    assert float(noise.median()) < 0.02


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_keys_just_inside_and_outside_the_chunks(tmp_root, dtype):
    """Prompts cut so that steps begin at, one before and one after the places where chunks and pages begin; then the
    same places decoded one by one."""
    from tq_kv_b200.engine import StepRow
    cfg = _chunk_cfg()
    path = pg.write_folder(os.path.join(str(tmp_root), "chunks"), cfg, make_weights(cfg, 9, sharp=True))
    eng = _engine(path, dtype)
    toks = tokens(200, cfg["vocab"], 13)
    want = oracle(path, toks)
    s = eng.new_sequence()
    _check(eng.step([StepRow(s, toks, list(range(200)))]), want, dtype, "chunks whole")
    eng.release(s)
    for cuts in ((63, 1, 1, 1, 4, 58, 1, 1, 1, 64, 5), (64, 6, 58, 6, 64, 2), (65, 64, 5, 1, 63, 2), (69, 1, 64, 64, 2)):
        assert sum(cuts) == 200
        s, at, got = eng.new_sequence(), 0, []
        for n in cuts:
            got.append(eng.step([StepRow(s, toks[at:at + n], list(range(n)))]))
            at += n
        _check(torch.cat(got), want, dtype, f"chunks, portions {cuts}")
        eng.release(s)
    s = eng.new_sequence()
    got = [eng.step([StepRow(s, toks[:60], [59])])]
    for t in range(60, 200):                                 # every edge is decoded alone
        got.append(eng.step([StepRow(s, [toks[t]], [0])]))
    _check(torch.cat(got), want[59:], dtype, "decoded across the chunks' edges")
    eng.release(s)


# ---- one set of tensors, two runs ----------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_a_layer_with_another_s_tensors_has_a_cache_and_a_state_of_its_own(tmp_root, dtype):
    """Both kinds of layer run twice in a row with one set of tensors: the same as two layers with equal tensors, and
    the memory that the second run keeps is not the first one's."""
    from tq_kv_b200.engine import StepRow
    one = {**delta(2, 1, 16, 16, 3), "mlp": dense(40)}
    two = {**both(2, 1, 16, 16, 40, 0.4, 24), "mlp": None}
    cfg = model(90, 64, 1e-6, 2, 0.9, 1.5, [one, {**one, "weights_of": 0}, two, {**two, "weights_of": 2}])
    w = make_weights(cfg, 4)
    path = pg.write_folder(os.path.join(str(tmp_root), f"twice_{dtype}"), cfg, w)
    toks = tokens(110, 90, 3)
    want = oracle(path, toks)
    w2 = {**w, **{n.replace(f"l{a}.", f"l{b}.", 1): t for n, t in w.items() for a, b in ((0, 1), (2, 3)) if n.startswith(f"l{a}.")}}
    plain = [dict(l) for l in cfg["layers"]]
    for l in plain:
        l.pop("weights_of", None)
    assert torch.equal(pg.decoder({**cfg, "layers": plain}, w2, toks), want.logits)
    eng = _engine(path, dtype)
    kv, state = eng.model.cache_requests()
    assert sorted(kv) == [2, 3] and sorted(state) == [0, 1, 2, 3] and len(eng.model.blocks) == 2
    s = eng.new_sequence()
    got = [eng.step([StepRow(s, toks[:60], list(range(60)))])]
    for t in range(60, 110):
        got.append(eng.step([StepRow(s, [toks[t]], [0])]))
    _check(torch.cat(got), want, dtype, "tensors used twice")
    assert not torch.equal(eng.cache.state[0][s], eng.cache.state[1][s])
    eng.release(s)


# ---- the entry points -------------------------------------------------------------------------------------------
def _same_or_tie(got, want, cfg, w, prompt):
    """Two logits may tie within float32 rounding: up to the first difference, which must be a tie."""
    n = next((i for i, (x, y) in enumerate(zip(got, want)) if x != y), len(want))
    if n < len(want):
        row = pg.decoder(cfg, w, prompt + want[:n])[-1]
        assert abs(float(row[got[n]] - row[want[n]])) < 1e-4 * float(row.abs().max()), (n, got, want)


def test_greedy_generation_through_the_entry_point_and_the_command_line(tmp_root):
    import tq_kv_b200 as tq
    path = folder(tmp_root, "c")
    cfg, w = pg.read_folder(path)
    prompts = [tokens(n, cfg["vocab"], 300 + n) for n in (3, 20, 9)]
    want = [pg.greedy(cfg, w, p, 10) for p in prompts]
    eng = tq.load(path, dtype="float32", max_batch=2, max_context=128)      # three requests, two slots
    res = eng.generate(prompts, tq.GenerationParams.greedy(10, stop_token_ids=()))
    assert all(r.finish_reason == "length" and len(r.tokens) == 10 for r in res)
    for r, wt, p in zip(res, want, prompts):
        _same_or_tie(r.tokens, wt, cfg, w, p)
    assert eng.cache.free_slots == 2
    env = dict(os.environ, PYTHONPATH=ROOT)
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "tq"), "run", path, "--dtype", "float32",
                        "--prompt-ids", ",".join(map(str, prompts[1])), "-n", "10", "--temperature", "0",
                        "--repeat-penalty", "1.0", "--max-context", "128"], capture_output=True, text=True, env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    _same_or_tie([int(t) for t in p.stdout.strip().splitlines()[-1].split(",")], want[1], cfg, w, prompts[1])


def test_greedy_generation_past_the_chunks_with_requests_that_wait_for_a_slot(tmp_root):
    """Five requests on two slots: each generates past several chunks; the scheduler gives freed slots, pages and
    states to the waiting ones."""
    import tq_kv_b200 as tq
    path = folder(tmp_root, "a")
    cfg, w = pg.read_folder(path)
    prompts = [tokens(n, cfg["vocab"], 400 + n) for n in (2, 70, 31, 5, 66)]
    want = [pg.greedy(cfg, w, p, 40, torch.float32) for p in prompts]
    eng = tq.load(path, dtype="float32", max_batch=2, max_context=192)
    res = eng.generate(prompts, tq.GenerationParams.greedy(40, stop_token_ids=()))
    for r, wt, p in zip(res, want, prompts):
        _same_or_tie(r.tokens, wt, cfg, w, p)
    assert eng.cache.free_slots == 2
    eng.cache.book.check()


def test_trace_replay_as_a_program(tmp_root, tmp_path):
    import numpy as np
    V = CASES["b"]["vocab"]
    a, b = tokens(100, V, 5), tokens(40, V, 6)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:90], "want": [0, 89]}, {"id": "y", "tokens": b[:38], "want": [37]}],
              "end": []}]
    for i in range(10):
        e = [{"id": "x", "tokens": [a[90 + i]], "want": [0]}]
        if i < 2:
            e.append({"id": "y", "tokens": [b[38 + i]], "want": [0] if i else []})
        steps.append({"step": i + 1, "entries": e, "end": ["y"] if i == 1 else (["x"] if i == 9 else [])})
    path = folder(tmp_root, "b")
    wa, wb = oracle(path, a), oracle(path, b)
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        p = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", path, "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "256"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                           capture_output=True, text=True, timeout=900)
        assert p.returncode == 0, p.stderr[-2000:]
        assert [l for l in p.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(11)]
        first = torch.from_numpy(np.fromfile(out / "0.f32", dtype="<f4").reshape(3, V).copy())
        _check(first, Want.cat([wa[0], wa[89], wb[37]]), dtype, "trace step 0")
        last = torch.from_numpy(np.fromfile(out / "10.f32", dtype="<f4").reshape(1, V).copy())
        _check(last, wa[99:100], dtype, "trace last step")
        two = torch.from_numpy(np.fromfile(out / "2.f32", dtype="<f4").reshape(2, V).copy())
        _check(two, Want.cat([wa[91], wb[39]]), dtype, "trace step 2")


def test_random_weights_from_a_named_shape(tmp_path):
    """`gokapel-tiny` with random weights: the engine made on the device and the folder written on the host hold the
    same weights, and the oracle agrees with both."""
    from tq_kv_b200.config import named_shape
    from tq_kv_b200.engine import Engine, StepRow
    from tq_kv_b200.weights import write_model_folder
    cfg = named_shape("gokapel-tiny")
    path = write_model_folder(cfg, str(tmp_path / "m"), 3)
    toks = tokens(90, cfg["vocab"], 4)
    want = oracle(path, toks)
    for eng in (Engine.from_random(cfg, 3, dtype="float32", max_tokens=256),
                Engine.from_folder(path, dtype="float32", max_tokens=256)):
        s = eng.new_sequence()
        _check(eng.step([StepRow(s, toks, list(range(90)))]), want, "float32", "named shape, random weights")
