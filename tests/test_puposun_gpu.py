"""The Puposun design on the GPU against its plain statement: whole models under every cutting, batches, slots and pages
used again, replayed steps, the engine's entry points, keys at the edges of windows, first tokens and far keys, and every
new or changed kernel alone."""
from __future__ import annotations

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import kernel_refs as R
import plain_puposun as pp
from helpers import cut, random_tokens, rel_err
from puposun_cases import CASE_A, CASE_B, CASES, experts, full, make_weights, model, random_case, windowed

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-4, torch.bfloat16: 3e-2}
SEEDS = {"A": 11, "B": 12, "C": 13, "D": 14}


def assert_close(got, want, dtype):
    """float32: every row within 2e-4 of its largest value.  bfloat16: where two experts' scores all but tie, rounding
    may choose the other one, so the rows are judged together: their median error and the ninth of ten."""
    if isinstance(got, (list, tuple)):                   # several requests: their rows are judged together
        got, want = torch.cat(list(got)), torch.cat(list(want))
    if dtype == torch.float32:
        assert rel_err(got, want) < TOL[dtype]
        return
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape and bool(torch.isfinite(got).all())
    err = (got - want).abs().amax(dim=1) / want.abs().amax(dim=1).clamp_min(1e-30)
    assert float(err.median()) < 1.2e-2, float(err.median())
    assert float(torch.quantile(err, 0.9)) < TOL[dtype], float(torch.quantile(err, 0.9))


def make_runner(case, w, dtype, n_pages=24, max_requests=3, page_size=16, use_graphs=False):
    from inferrs_b200.engine.loading import spec_from_config
    from inferrs_b200.engine.runner import ModelRunner
    from inferrs_b200.runtime import Runtime
    spec, _ = spec_from_config(case)
    rt = Runtime.cuda(dtype)
    return ModelRunner(spec, {k: v.to(dtype).cuda() for k, v in w.items()}, rt, page_size=page_size, n_pages=n_pages,
                       max_requests=max_requests, use_graphs=use_graphs)


def entry(rid, tokens, want=None):
    from inferrs_b200.engine.batch import StepEntry
    return StepEntry(rid, tokens, list(range(len(tokens))) if want is None else want)


def dev(v, dtype=torch.int32):
    return torch.tensor(v, dtype=dtype, device="cuda")


def act(x, dtype):
    return x.to(dtype).cuda().contiguous()


# ---------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_whole_prompt_and_every_cutting_match_the_plain_statement(name, dtype):
    case, w = CASES[name], make_weights(CASES[name], SEEDS[name])
    toks = random_tokens(110, case["vocab"], seed=3)
    want = pp.forward(case, w, toks)
    runner = make_runner(case, w, dtype)
    runner.admit("whole")
    assert_close(runner.step([entry("whole", toks)]), want, dtype)
    runner.release("whole")
    # one token a step from an empty cache: the first tokens of a sequence, and decoding through the cache
    runner.admit("single")
    rows = [runner.step([entry("single", [t])]) for t in toks[:90]]
    assert_close(torch.cat(rows), want[:90], dtype)
    runner.release("single")
    # portions of changing size, down to two tokens and one, another request's portions beside them
    other = random_tokens(40, case["vocab"], seed=4)
    want_other = pp.forward(case, w, other)
    runner.admit("cut")
    runner.admit("other")
    at, o_at, rows, o_rows = 0, 0, [], []
    for n in cut(len(toks), [7, 2, 30, 1, 1, 2, 17, 3]):
        entries = [entry("cut", toks[at:at + n])]
        if o_at < len(other):
            entries.insert(o_at % 2, entry("other", other[o_at:o_at + 6]))
        out = runner.step(entries)
        k = 0
        for e in entries:
            (rows if e.rid == "cut" else o_rows).append(out[k:k + len(e.tokens)])
            k += len(e.tokens)
        o_at += 6
        at += n
    assert_close(torch.cat(rows), want, dtype)
    assert_close(torch.cat(o_rows), want_other[:sum(r.shape[0] for r in o_rows)], dtype)
    runner.manager.check_invariants()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", list(range(14)))
def test_configurations_drawn_at_random(seed, dtype):
    """Sizes, counts, windows, constants, the order of layers and the loop drawn from a seed: a whole prompt, then the same
    prompt in portions with its last tokens one by one, in pages that the first request has used."""
    case = random_case(seed)
    w = make_weights(case, 100 + seed)
    toks = random_tokens(100, case["vocab"], seed=seed)
    want = pp.forward(case, w, toks)
    runner = make_runner(case, w, dtype, n_pages=8, max_requests=1)
    runner.admit("whole")
    assert_close(runner.step([entry("whole", toks)]), want, dtype)
    runner.release("whole")
    runner.admit("cut")
    rows, at = [], 0
    for n in cut(70, [19, 2, 33, 1, 5]):
        rows.append(runner.step([entry("cut", toks[at:at + n])]))
        at += n
    for t in toks[70:]:
        rows.append(runner.step([entry("cut", [t])]))
    assert_close(torch.cat(rows), want, dtype)
    runner.manager.check_invariants()


def test_the_stream_matches_after_every_layer_run():
    """What every layer run hands on, through the model's own blocks, in float32: models whose schedule ends after it."""
    from dataclasses import replace
    from inferrs_b200.engine.loading import spec_from_config
    from inferrs_b200.engine.runner import ModelRunner
    from inferrs_b200.runtime import Runtime
    case, w = CASE_A, make_weights(CASE_A, 17)
    toks = random_tokens(33, case["vocab"], seed=9)
    after = []
    pp.forward(case, w, toks, after_layers=after)
    spec, _ = spec_from_config(case)
    rt = Runtime.cuda(torch.float32)
    assert len(after) == len(spec.schedule)
    for upto in range(1, len(after) + 1):
        r = ModelRunner(replace(spec, schedule=spec.schedule[:upto]), {k: v.cuda() for k, v in w.items()}, rt, page_size=16,
                        n_pages=8, max_requests=1, use_graphs=False)
        r.admit(0)
        want = pp.squashed(pp.norm(after[upto - 1], w["final.norm"], case["norm"]["eps"]) @ w["head"].T, case["logit_softcap"])
        assert rel_err(r.step([entry(0, toks)]), want) < TOL[torch.float32], upto


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_unequal_requests_in_one_batch_slots_and_pages_used_again(name, dtype):
    """Two slots and pages for two requests; five requests of unequal length take turns, decoding side by side with
    portions of the next ones.  Every request must give what it gives alone (the plain statement knows no batches,
    slots or pages)."""
    case, w = CASES[name], make_weights(CASES[name], SEEDS[name])
    lens = {"a": 50, "b": 23, "c": 64, "d": 9, "e": 37}
    toks = {k: random_tokens(n, case["vocab"], seed=100 + ord(k)) for k, n in lens.items()}
    want = {k: pp.forward(case, w, t) for k, t in toks.items()}
    runner = make_runner(case, w, dtype, n_pages=9, max_requests=2)      # 144 cached tokens: no three requests fit
    got = {k: [] for k in lens}
    at = {k: 0 for k in lens}
    live, waiting = [], list(lens)
    sizes = [13, 1, 1, 2, 5, 1, 30, 1]
    i = 0
    while live or waiting:
        while waiting and len(live) < 2:
            k = waiting.pop(0)
            runner.admit(k)
            live.append(k)
        entries = []
        for j, k in enumerate(live):
            n = min(sizes[(i + 3 * j) % len(sizes)], lens[k] - at[k])
            entries.append(entry(k, toks[k][at[k]:at[k] + n]))
        out = runner.step(entries)
        r = 0
        for e in entries:
            got[e.rid].append(out[r:r + len(e.tokens)])
            r += len(e.tokens)
            at[e.rid] += len(e.tokens)
            if at[e.rid] == lens[e.rid]:
                runner.release(e.rid)
                live.remove(e.rid)
        i += 1
        runner.manager.check_invariants()
    assert_close([torch.cat(got[k]) for k in lens], [want[k] for k in lens], dtype)


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_replayed_steps_give_what_plain_launches_give(name):
    """The same requests through steps captured as CUDA graphs (padding requests without pages) and through steps
    launched kernel by kernel."""
    case, w = CASES[name], make_weights(CASES[name], SEEDS[name])
    toks = {k: random_tokens(n, case["vocab"], seed=n) for k, n in (("a", 70), ("b", 45), ("c", 20))}
    outs = []
    for graphs in (False, True):
        runner = make_runner(case, w, torch.bfloat16, use_graphs=graphs)
        assert (runner.graphs is not None) == graphs
        for k in "abc":
            runner.admit(k)
        rows = [runner.step([entry("a", toks["a"][:40]), entry("b", toks["b"][:33]), entry("c", toks["c"][:1])])]
        for i in range(12):
            rows.append(runner.step([entry("a", [toks["a"][40 + i]]), entry("c", [toks["c"][1 + i]]),
                                     entry("b", [toks["b"][33 + i]])]))
        rows.append(runner.step([entry("a", toks["a"][52:])]))
        outs.append(torch.cat(rows))
    assert_close(outs[1], outs[0], torch.bfloat16)
    want = torch.cat([pp.forward(case, w, toks["a"])[:40], pp.forward(case, w, toks["b"])[:33]])
    assert_close(outs[1][:73], want, torch.bfloat16)


@pytest.mark.parametrize("name", ["A", "C"])
def test_long_decoding_through_windows_and_kept_tokens(name):
    """Two hundred and more decoded tokens in replayed steps: windows pass over decoded tokens, their pages go back, the
    first tokens' pages stay."""
    case, w = CASES[name], make_weights(CASES[name], 21)
    toks = random_tokens(260, case["vocab"], seed=8)
    want = pp.forward(case, w, toks)
    runner = make_runner(case, w, torch.float32, n_pages=20, max_requests=1, use_graphs=True)
    runner.admit(0)
    rows = [runner.step([entry(0, toks[:5])])]
    for t in toks[5:]:
        rows.append(runner.step([entry(0, [t])]))
    assert rel_err(torch.cat(rows), want) < TOL[torch.float32]
    # pages that a window has passed are free again, those of its first tokens are not
    for g, layout in enumerate(runner.manager.groups):
        if layout.window:
            table = runner.manager.block_table(0, g)
            first = -(-layout.keep_first // 16)
            dead = max((260 - layout.window + 1) // 16, first)
            assert all(p >= 0 for p in table[:first]) and all(p < 0 for p in table[first:dead]) and all(p >= 0 for p in table[dead:])
    # the early tokens matter to the last logits: without them the far keys are other ones
    assert rel_err(pp.forward(case, w, toks[120:])[-1], want[-1]) > 1e-3


# ---------------------------------------------------------------------------------------------------
# through the engine's own entry points
# ---------------------------------------------------------------------------------------------------
def write_folder(path, case, w):
    from inferrs_b200.weights.safetensors_io import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(case, f)
    write_safetensors(os.path.join(path, "model.safetensors"), [(k, v.to(torch.bfloat16)) for k, v in w.items()])
    return path


def test_greedy_generation_through_the_engine(tmp_path):
    """More requests than slots and few pages: the scheduler admits, cuts prompts into portions, preempts and computes
    again; every request gets the tokens that the plain statement picks."""
    from inferrs_b200.engine.engine import Engine
    from inferrs_b200.sampling.params import SamplingParams
    case, w = CASE_A, make_weights(CASE_A, 31)
    folder = write_folder(str(tmp_path / "m"), case, w)
    eng = Engine(model_dir=folder, dtype="f32", block_size=16, num_blocks=8, max_batch_size=2, max_tokens_per_step=24)
    prompts = [random_tokens(n, case["vocab"], seed=60 + n) for n in (33, 5, 40, 18)]
    n_new = 12
    want = [pp.greedy(case, w, p, n_new) for p in prompts]
    got = eng.generate(prompts, SamplingParams.greedy(max_tokens=n_new))
    eng.runner.manager.check_invariants()
    assert got == want
    assert eng.generate(prompts[:2], SamplingParams.greedy(max_tokens=n_new)) == want[:2]    # slots used before


def test_command_line_with_random_weights_and_with_a_folder(tmp_path, capsys):
    from inferrs_b200 import cli
    path = str(tmp_path / "config.json")
    with open(path, "w") as f:
        json.dump(dict(CASE_A, eos_token_id=5), f)
    common = [path, "--random-weights", "4", "--max-blocks", "32", "--max-batch-size", "2", "--max-tokens", "7",
              "--ignore-eos", "--seed", "3", "--prefill-chunk", "16", "--random-prompt", "45"]
    outs = []
    for _ in range(2):
        assert cli.main(["run"] + common + ["--temperature", "0.8", "--top-k", "20", "--dtype", "bf16"]) == 0
        cap = capsys.readouterr()
        outs.append([int(t) for t in cap.out.split()])
        assert "45 prompt tokens, 7 generated" in cap.err
    assert outs[0] == outs[1] and len(outs[0]) == 7 and all(0 <= t < CASE_A["vocab"] for t in outs[0])
    folder = write_folder(str(tmp_path / "m"), CASE_B, make_weights(CASE_B, 5))
    assert cli.main(["bench", folder, "--prompt-len", "30", "--max-tokens", "6", "--runs", "2", "--warmup", "1",
                     "--max-blocks", "32", "--max-batch-size", "2", "--temperature", "0"]) == 0
    out = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert out["prompt_len"] == 30 and out["prefill_tok_s"] > 0 and out["decode_tok_s"] > 0


def test_trace_replay_of_a_folder(tmp_path):
    """A later request takes the slot and the pages of one that ended."""
    case, w = CASE_A, make_weights(CASE_A, 41)
    folder = write_folder(str(tmp_path / "m"), case, w)
    toks = {k: random_tokens(n, case["vocab"], seed=n) for k, n in (("a", 70), ("b", 21), ("c", 30))}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks["a"][:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks["a"][50:51], "want": [0]},
                                     {"id": "b", "tokens": toks["b"][:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": toks["b"][19:], "want": [0, 1]},
                                     {"id": "a", "tokens": toks["a"][51:], "want": [18]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": toks["c"][:28], "want": []}], "end": []},
             {"step": 4, "entries": [{"id": "c", "tokens": toks["c"][28:], "want": [0, 1]}], "end": ["c"]}]
    out_dir = str(tmp_path / "out")
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32",
                        "--out", out_dir, "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert p.returncode == 0, p.stderr[-800:]
    assert p.stdout.split() == ["done", "0", "done", "1", "done", "2", "done", "3", "done", "4"]
    wa, wb, wc = (pp.forward(case, w, toks[k]) for k in "abc")
    read = lambda s: torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{s}.f32"), dtype="<f4").reshape(-1, case["vocab"]).copy())   # noqa: E731
    assert rel_err(read(0), wa[[0, 49]]) < 2e-4
    assert rel_err(read(1), torch.stack([wa[50], wb[18]])) < 2e-4
    assert rel_err(read(2), torch.stack([wb[19], wb[20], wa[69]])) < 2e-4
    assert not os.path.exists(os.path.join(out_dir, "3.f32"))
    assert rel_err(read(4), wc[[28, 29]]) < 2e-4


# ---------------------------------------------------------------------------------------------------
# single keys that stand out, in the model: weights under which a token's id is its query and key
# ---------------------------------------------------------------------------------------------------
W64 = 64
ASK, MARK, CHANNEL = 7, 9, -1          # the token that asks, the token it asks for, and the head's number that carries both


def story(layer):
    """One layer under whose weights only token ASK has a query and only token MARK a key (the same last number of a
    head, which does not turn); the value, being the key, is the mark itself and reaches channel 60 of the stream.  The
    embedding is the identity, the norms divide and do no more, logits are the last norm's rows (the cap is far away)."""
    case = model(W64, W64, 1e-5, 8.0, 1000.0, [layer])
    m = layer["mixer"]
    w = {k: torch.zeros_like(v) for k, v in make_weights(case, 7).items()}
    w["embed"], w["head"] = torch.eye(W64), torch.eye(W64)
    w["l0.norm1"], w["final.norm"] = torch.ones(W64), torch.ones(W64)
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    w["l0.mix.q"].view(H, D, W64)[:, CHANNEL, ASK] = 1.0
    w["l0.mix.k"].view(G, D, W64)[:, CHANNEL, MARK] = 1.0
    w["l0.mix.o"].view(W64, H, D)[60, :, CHANNEL] = 1.0 / H
    return case, w


def run_whole_and_cut(case, w, dtype, toks, portions, single_from, single_to, use_graphs=False):
    """The logits of the whole prompt in one step, and of the same prompt in portions with the tokens
    single_from..single_to decoded one by one (a request after the whole one, in a slot and pages that it used)."""
    runner = make_runner(case, w, dtype, n_pages=60, max_requests=2, use_graphs=use_graphs)
    runner.admit("w")
    got = runner.step([entry("w", toks)])
    runner.release("w")
    runner.admit("c")
    rows, at = [], 0
    for k in cut(single_from, portions):
        rows.append(runner.step([entry("c", toks[at:at + k])]))
        at += k
    for t in toks[single_from:single_to]:
        rows.append(runner.step([entry("c", [t])]))
    if single_to < len(toks):
        rows.append(runner.step([entry("c", toks[single_to:])]))
    return got, torch.cat(rows)


def background(n):
    """Tokens that neither ask nor are asked for."""
    return [(11 + 3 * i) % 40 + 12 for i in range(n)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,marked_at,heads,kv,dim", [(37, 0, 200, 2, 1, 32), (48, 3, 208, 4, 2, 64), (5, 16, 203, 6, 2, 128),
                                                              (64, 17, 192, 3, 3, 24), (1, 1, 150, 2, 2, 16), (65, 64, 127, 8, 2, 128),
                                                              (33, 70, 191, 4, 4, 96)])
def test_a_marked_token_is_seen_inside_the_window_and_not_beyond(size, keep, marked_at, heads, kv, dim, dtype):
    """MARK stands once in a prompt of other tokens; ASK asks for it at every distance around the window's edge, in a
    whole prompt, in portions and decoded one by one.  It is found while it is inside the window and not one token later
    (the kept first tokens are long past)."""
    case, w = story(windowed(heads, kv, dim, 4, 100.0, 0.25, size, keep))
    n = marked_at + size + 12
    toks = background(n)
    toks[marked_at] = MARK
    asks = list(range(marked_at + max(size - 4, 1), marked_at + size + 3))
    for a in asks:
        toks[a] = ASK
    want = pp.forward(case, w, toks)
    for a in asks:
        assert (float(want[a, 60]) > 3.0) == (a - marked_at < size), (a, float(want[a, 60]))
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], marked_at + max(size - 2, 1), n - 2)
    tol = 2e-4 if dtype == torch.float32 else 3e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep,dim", [(20, 1, 16), (16, 15, 64), (33, 16, 128), (64, 17, 128), (7, 64, 96), (40, 65, 128),
                                           (70, 130, 128), (9, 5, 24)])
@pytest.mark.parametrize("inside", [True, False])
def test_the_last_kept_token_is_seen_from_everywhere_and_the_next_one_is_not(inside, size, keep, dim, dtype):
    """MARK stands on the last kept place or on the one behind it; ASK asks from inside the window, from just beyond it
    and from hundreds of tokens later (long after the pages between have gone back)."""
    case, w = story(windowed(4, 2, dim, 4, 100.0, 0.25, size, keep))
    at = keep - 1 if inside else keep
    n = at + size + 300
    toks = background(n)
    toks[at] = MARK
    asks = [at + 1, at + size - 1, at + size, at + size + 1, at + size + 90, n - 20, n - 1]
    for a in asks:
        if a > at:
            toks[a] = ASK
    want = pp.forward(case, w, toks)
    for a in asks:
        if a > at:
            assert (float(want[a, 60]) > 3.0) == (inside or a - at < size), (a, float(want[a, 60]))
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], n - 30, n - 1, use_graphs=True)
    tol = 2e-4 if dtype == torch.float32 else 3e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv,dim,marked_at", [(4, 2, 64, 15), (2, 1, 128, 16), (6, 3, 24, 255), (8, 2, 128, 0), (5, 5, 80, 127),
                                                    (3, 1, 96, 64)])
def test_a_marked_token_far_back_is_found_among_hundreds(heads, kv, dim, marked_at, dtype):
    """Every earlier key visible: a marked token hundreds of positions back, just before and just after a page's border
    and at the very start, is found by the token that asks for it and by no other.  Its score is 16, squashed by a cap
    of 20; without the cap the share of the others would be another one, which the capped value shows."""
    case, w = story(full(heads, kv, dim, 4, 100.0, 0.25, 20.0))
    n = 400
    toks = background(n)
    toks[marked_at] = MARK
    asks = (marked_at + 1, 300, 399)
    for a in asks:
        toks[a] = ASK
    want = pp.forward(case, w, toks)
    assert all(float(want[a, 60]) > 3.0 for a in asks) and float(want[298, 60]) < 1.0 and float(want[398, 60]) < 1.0
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], 290, 310)
    tol = 2e-4 if dtype == torch.float32 else 3e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap", [2.0, 20.0])
@pytest.mark.parametrize("heads,kv,dim", [(2, 1, 32), (4, 2, 128), (6, 6, 20), (8, 2, 64)])
def test_cap_and_sink_decide_the_share_of_a_key(heads, kv, dim, cap, dtype):
    """Everybody's key is the same, with a score that the cap squashes (3.2, to 1.84 or 3.17): at position i every one of the i + 1 keys has
    the share e^s / (1 + (i + 1) e^s), so the value that comes out tells cap and sink at the first tokens, where the
    sink weighs most, and hundreds of tokens on."""
    case, w = story(full(heads, kv, dim, 4, 100.0, 0.05, cap))
    w["l0.mix.q.b"].view(heads, dim)[:, CHANNEL] = 8.0
    w["l0.mix.k"].zero_()
    w["l0.mix.k.b"].view(kv, dim)[:, CHANNEL] = 8.0          # the value is the key with its bias
    toks = background(330)
    want = pp.forward(case, w, toks)
    s = cap * np.tanh(3.2 / cap)
    for i in (0, 1, 2, 300):
        share = (i + 1) * np.exp(s) / (1 + (i + 1) * np.exp(s))
        x60 = 8.0 * share
        assert abs(float(want[i, 60]) - x60 / np.sqrt((64 + x60 * x60) / 64 + 1e-5)) < 1e-3
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [1, 1, 2, 50, 7, 2, 64, 3], 300, 325)
    tol = 2e-4 if dtype == torch.float32 else 1e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol
    assert rel_err(got[:3], want[:3]) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind,rot,dim", [("halves", 16, 32), ("neighbours", 16, 32), ("halves", 64, 128), ("neighbours", 128, 128),
                                          ("neighbours", 8, 64), ("halves", 14, 19)])
@pytest.mark.parametrize("back", [0, 1, 17, 63])
def test_the_rotation_finds_a_token_by_its_distance(back, kind, rot, dim, dtype):
    """Every token's key is the same before it is turned and the query is that key turned ``back`` positions the other
    way: each token finds the one exactly that far back, and takes its value, which is its key before it is turned."""
    layer = full(2, 1, dim, rot, 40.0, 1.0, 60.0) if kind == "halves" else windowed(2, 1, dim, rot, 40.0, 1.0, 400, 0)
    case, w = story(layer)
    turn = pp.rotate_halves if kind == "halves" else pp.rotate_neighbours
    base = torch.zeros(1, 1, dim)
    if kind == "halves":
        base[0, 0, :rot // 2] = 1.0
    else:
        base[0, 0, 0:rot:2] = 1.0
    base *= (24.0 / rot) ** 0.5
    ask = turn(base, torch.tensor([-back]), 40.0, rot)[0, 0]
    for name, vec, heads in (("q", ask, 2), ("k", base[0, 0], 1)):
        t = w[f"l0.mix.{name}"].zero_().view(heads, dim, W64)
        t += vec[None, :, None] / 8.0                             # every token's normed row is 8 in one place
    # what the value says: the marked token has a further number, which does not turn (or, where all turn, a little more)
    if dim > rot:
        w["l0.mix.k"].view(1, dim, W64)[0, -1, MARK] = 1.0
        w["l0.mix.q"].view(2, dim, W64)[:, -1] = 0.0
    else:
        w["l0.mix.k"].view(1, dim, W64)[0, -1, MARK] = 0.25
    n = 330
    toks = background(n)
    for i in (3, 100, 250, 320 - back):
        toks[i] = MARK
    want = pp.forward(case, w, toks)
    found = [i for i in range(back, n) if float(want[i, 60]) > 0.5 * float(want[:, 60].max())]
    assert set(p + back for p in (100, 250, 320 - back)) <= set(found) and len(found) < 40
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], 300, 325)
    tol = 2e-4 if dtype == torch.float32 else 6e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


# ---------------------------------------------------------------------------------------------------
# the attention kernels alone, with every option that each of them takes
# ---------------------------------------------------------------------------------------------------
class Step:
    """A batch of unequal requests over shuffled pages that hold no numbers where no request owns them."""

    def __init__(self, held, lens, nh, nkv, d, page, dtype, seed, window, keep):
        g = torch.Generator().manual_seed(seed)
        self.lens, self.held, n = lens, held, sum(lens)
        total = [a + b for a, b in zip(held, lens)]
        need = [(t + page - 1) // page for t in total]
        order = torch.randperm(sum(need) + 3, generator=g).tolist()
        k_pages = torch.full((len(order), nkv, page, d), float("nan"))
        v_pages = torch.full((len(order), nkv, page, d), float("nan"))
        table = torch.full((len(lens), max(need) + 1), -1, dtype=torch.int32)
        for r, t in enumerate(total):
            keys, values = torch.randn(t, nkv, d, generator=g), torch.randn(t, nkv, d, generator=g)
            for p in range(need[r]):
                # pages that the window has passed for every row of the step, and that hold no kept key, are gone
                if window and (p + 1) * page <= held[r] - window + 1 and p * page >= keep:
                    continue
                table[r, p] = pid = order.pop()
                k_pages[pid] = 0.0
                v_pages[pid] = 0.0
                part = slice(p * page, min((p + 1) * page, t))
                k_pages[pid, :, :part.stop - part.start] = keys[part].transpose(0, 1)
                v_pages[pid, :, :part.stop - part.start] = values[part].transpose(0, 1)
        self.k, self.v, self.table = act(k_pages, dtype), act(v_pages, dtype), table.cuda()
        self.q = act(torch.randn(n, nh, d, generator=g), dtype)
        self.positions = dev([a + i for a, b in zip(held, lens) for i in range(b)])
        self.row_request = dev([r for r, b in enumerate(lens) for _ in range(b)])
        self.q_start = dev([0] + list(np.cumsum(lens)))
        self.gate = act(torch.randn(n, nh + 5, generator=g) * 2, dtype)
        self.head = {"head_scale": 1 + 0.5 * torch.randn(nh, generator=g), "slopes": 0.05 * torch.rand(nh, generator=g),
                     "sinks": torch.randn(nh, generator=g)}

    def options(self, names, keep):
        opt = {k: self.head[k].cuda() for k in ("head_scale", "slopes", "sinks") if k in names}
        if "cap" in names:
            opt["cap"] = 2.5
        if keep:
            opt["keep_first"] = keep
        if "gate" in names:
            opt["gate"] = self.gate[:, 3:]
        return opt

    def tiles(self, tokens):
        t = [(-1, 0)] + [(r, int(self.q_start[r]) + i) for r, n in enumerate(self.lens) for i in range(0, n, tokens)]
        return dev([a for a, _ in t]), dev([b for _, b in t]), len(t)

    def want(self, scale, window, options):
        out = torch.empty(self.q.shape[0], self.q.shape[1] * self.q.shape[2])
        cpu = {k: (v.float().cpu() if isinstance(v, torch.Tensor) else v) for k, v in options.items()}
        R.paged_attention_generic(self.q.float().cpu(), self.k.float().cpu(), self.v.float().cpu(), self.table.cpu(),
                                  self.row_request.cpu(), self.positions.cpu(), scale, window, out, **cpu)
        return out


def wide_out(n, cols, dtype, extra=24, first=8):
    """Rows that lie further apart than they are long; what lies between them must stay as it is."""
    whole = torch.full((n, cols + extra), 7.0, dtype=dtype, device="cuda")
    return whole, whole[:, first:first + cols]


ALL = ("head_scale", "slopes", "sinks", "cap", "gate")
OPTIONS = [(), ("cap",), ("sinks", "cap"), ("gate",), ALL]
WINDOWS = [(None, 0), (64, 0), (37, 5), (65, 16), (16, 70), (130, 129), (1, 1)]


def check_out(whole, out, first, want, dtype):
    assert rel_err(out.float(), want) < (2e-5 if dtype == torch.float32 else 2.5e-2)
    assert bool((whole[:, :first] == 7.0).all()) and bool((whole[:, first + out.shape[1]:] == 7.0).all())


@pytest.mark.parametrize("names", OPTIONS, ids=lambda o: "+".join(o) or "plain")
@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("dtype", DTYPES)
def test_generic_attention_with_options(dtype, window, keep, names):
    from inferrs_b200 import kernels as K
    for nh, nkv, d, page in ((6, 2, 20, 16), (3, 3, 48, 8)):
        s = Step([0, 150, 31], [40, 1, 5], nh, nkv, d, page, dtype, 3, window, keep)
        opt = s.options(names, keep)
        whole, out = wide_out(46, nh * d, dtype)
        K.paged_attention_generic(s.q, s.k, s.v, s.table, s.row_request, s.positions, 0.3, window, out, **opt)
        check_out(whole, out, 8, s.want(0.3, window, opt), dtype)


@pytest.mark.parametrize("names", OPTIONS, ids=lambda o: "+".join(o) or "plain")
@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("d", [32, 80, 96, 128, 192])
def test_mma_attention_with_options(d, window, keep, names):
    from inferrs_b200 import kernels as K
    bf = torch.bfloat16
    nh, nkv = (6, 2) if d != 96 else (5, 1)
    s = Step([0, 150, 31], [70, 2, 33], nh, nkv, d, 16, bf, 4, window, keep)
    opt = s.options(names, keep)
    whole, out = wide_out(105, nh * d, bf)
    req, row0, n_tiles = s.tiles(K.MMA_KEYS // (nh // nkv))
    K.paged_attention_mma(s.q, s.k, s.v, s.table, req, row0, n_tiles, s.q_start, s.positions, 0.2, window, out, False, **opt)
    check_out(whole, out, 8, s.want(0.2, window, opt), bf)
    # single tokens, keys in one piece and cut over three and eight CTAs
    s = Step([0, 700, 31, 64, 255], [1] * 5, nh, nkv, d, 16, bf, 5, window, keep)
    opt = s.options(names, keep)
    want = s.want(0.2, window, opt)
    for splits in (1, 3, 8):
        whole, out = wide_out(5, nh * d, bf)
        K.paged_attention_mma(s.q, s.k, s.v, s.table, s.row_request, s.q_start, 5, s.q_start, s.positions, 0.2, window, out, True,
                              splits, **opt)
        check_out(whole, out, 8, want, bf)


@pytest.mark.parametrize("names", OPTIONS, ids=lambda o: "+".join(o) or "plain")
@pytest.mark.parametrize("window,keep", WINDOWS)
@pytest.mark.parametrize("nh,nkv", [(8, 2), (5, 1), (4, 4)])
def test_tma_and_tcgen05_attention_with_options(nh, nkv, window, keep, names):
    """The decode kernel (one and several slices, a list of rows), the tcgen05 kernel in its three forms, and the one
    with two query tiles, which takes kept keys and the gate."""
    from inferrs_b200 import kernels as K
    bf, d = torch.bfloat16, 128
    s = Step([0, 700, 31, 64, 255], [1] * 5, nh, nkv, d, 16, bf, 6, window, keep)
    opt = s.options(names, keep)
    want = s.want(0.09, window, opt)
    for splits, min_tiles in ((1, 4), (3, 1), (12, 1)):
        whole, out = wide_out(5, nh * d, bf)
        K.paged_attention_decode(s.q, s.k, s.v, s.table, s.positions, 0.09, window, out, splits, min_tiles=min_tiles, **opt)
        check_out(whole, out, 8, want, bf)
    whole, out = wide_out(5, nh * d, bf)
    K.paged_attention_decode(s.q, s.k, s.v, s.table, s.positions, 0.09, window, out, 3, dev([3, -1, 1]), dev([3, -1, 1]), min_tiles=1,
                             **opt)
    check_out(whole[[1, 3]], out[[1, 3]], 8, want[[1, 3]], bf)
    assert bool((out[[0, 2, 4]] == 7.0).all()) and K.attention_decode_error() == 0
    s = Step([0, 300, 31], [200, 70, 2], nh, nkv, d, 16, bf, 7, window, keep)
    opt = s.options(names, keep)
    want = s.want(0.09, window, opt)
    req, row0, n_tiles = s.tiles(K.TC_ROWS // (nh // nkv))
    whole, out = wide_out(272, nh * d, bf)
    K.paged_attention_tcgen05(s.q, s.k, s.v, s.table, req, row0, n_tiles, s.q_start, s.positions, 0.09, window, out, **opt)
    check_out(whole, out, 8, want, bf)
    assert K.attention_tcgen05_error() == 0
    if not K.ScoreOptions(**opt).shape_scores:
        req, row0, n_tiles = s.tiles(K.pair_tile_tokens(nh, nkv))
        whole, out = wide_out(272, nh * d, bf)
        K.paged_attention_pair_tcgen05(s.q, s.k, s.v, s.table, req, row0, n_tiles, s.q_start, s.positions, 0.09, window, out, **opt)
        check_out(whole, out, 8, want, bf)
        assert K.attention_pair_tcgen05_error() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [24, 64, 128])
def test_kept_keys_stand_out_at_every_border(d, dtype):
    """One key is made to stand out, so that whoever sees it gives its value alone: on the last kept place and the one
    behind it, at borders of pages and of key tiles, just inside and just outside the window, from single rows and from
    prompt portions (whichever kernel the step's dispatch picks)."""
    from inferrs_b200 import kernels as K
    nh, nkv, page, T = 4, 2, 16, 420
    g = torch.Generator().manual_seed(d)
    for j, pos, window, keep in ((4, 400, 20, 5), (5, 400, 20, 5), (15, 300, 64, 16), (16, 300, 64, 16), (63, 410, 33, 64),
                                 (64, 410, 33, 64), (127, 399, 70, 128), (128, 399, 70, 128), (0, 419, 1, 1), (1, 419, 1, 1),
                                 (380, 400, 21, 5), (379, 400, 21, 5), (69, 100, 40, 70), (61, 100, 40, 10), (60, 100, 40, 10),
                                 (100, 100, 40, 10), (3, 3, 40, 2)):
        keys, values = torch.zeros(T, nkv, d), torch.randn(T, nkv, d, generator=g).to(dtype).float()
        keys[j] = 4.0 / d ** 0.5
        order = torch.randperm(30, generator=g).tolist()
        k_pages, v_pages = torch.full((30, nkv, page, d), float("nan")), torch.full((30, nkv, page, d), float("nan"))
        table = torch.full((1, 28), -1, dtype=torch.int32)
        for p in range((T + page - 1) // page):
            if (p + 1) * page <= pos - 9 - window + 1 and p * page >= keep:
                continue
            table[0, p] = pid = order[p]
            part = slice(p * page, min((p + 1) * page, T))
            k_pages[pid], v_pages[pid] = 0.0, 0.0
            k_pages[pid, :, :part.stop - part.start] = keys[part].transpose(0, 1)
            v_pages[pid, :, :part.stop - part.start] = values[part].transpose(0, 1)
        q = torch.full((10, nh, d), 12.0 / d ** 0.5)
        seen = j <= pos and (pos - j < window or j < keep)
        see = [i for i in range(pos + 1) if pos - i < window or i < keep]
        want = (values[j] if seen else values[see].mean(0)).repeat_interleave(nh // nkv, dim=0).reshape(nh * d)

        class Ctx:
            decode_only, n_rows, n_requests, max_kv_len, extra = True, 1, 1, 420, {}

        for first in ((pos,), tuple(range(max(pos - 9, 0), pos + 1))):
            n = len(first)
            ctx = Ctx()
            ctx.decode_only, ctx.n_rows, ctx.extra = n == 1, n, {}
            ctx.positions, ctx.row_request, ctx.q_start = dev(list(first)), dev([0] * n), dev([0, n])
            ctx.attention_tiles = lambda tokens, portions_only=False: (
                dev([0] * len(range(0, n, tokens))), dev(list(range(0, n, tokens))), len(range(0, n, tokens)))
            ctx.single_rows = lambda: (dev([]), dev([]), 0)
            out = torch.empty(n, nh * d, dtype=dtype, device="cuda")
            K.paged_attention(act(q[:n], dtype), act(k_pages, dtype), act(v_pages, dtype), table.cuda(), ctx, 1.0, window, out,
                              keep_first=keep)
            assert rel_err(out[-1:].float(), want[None]) < (1e-5 if dtype == torch.float32 else 3e-2), (j, pos, window, keep, n)


# ---------------------------------------------------------------------------------------------------
# the other kernels alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("biased", [False, True])
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("nh,nkv,d,rot", [(6, 2, 24, 16), (4, 4, 16, 8), (5, 1, 11, 6), (8, 2, 128, 128), (3, 3, 64, 0), (16, 4, 96, 48),
                                          (2, 1, 30, 14), (7, 7, 80, 80), (4, 2, 32, 4)])
def test_values_that_are_keys_are_stored_before_they_turn(nh, nkv, d, rot, interleaved, biased, dtype):
    from inferrs_b200 import kernels as K
    g = torch.Generator().manual_seed(nh * d)
    lens, held, page = [9, 1, 20, 3], [30, 64, 0, 15], 16
    n = sum(lens)
    cols = (nh + nkv) * d
    for extra in (0, 8, 13):                              # columns behind the keys, which nobody reads
        qkv = torch.randn(n, cols + extra, generator=g).to(dtype)
        bias = torch.randn(cols, generator=g) if biased else None
        need = [(a + b + page - 1) // page for a, b in zip(lens, held)]
        order = torch.randperm(sum(need) + 2, generator=g).tolist()
        table = torch.full((4, max(need) + 1), -1, dtype=torch.int32)
        for r, k in enumerate(need):
            table[r, :k] = torch.tensor([order.pop() for _ in range(k)], dtype=torch.int32)
        table[1, 64 // page] = -1                          # a request without a page there: nothing is written
        k_pages = torch.full((sum(need) + 2, nkv, page, d), 5.0, dtype=dtype, device="cuda")
        v_pages = torch.full_like(k_pages, 5.0)
        positions = [h + i for h, k in zip(held, lens) for i in range(k)]
        req = [r for r, k in enumerate(lens) for _ in range(k)]
        cos = sin = None
        if rot:
            c, s = pp.angles(torch.arange(200), 100.0, rot)
            cos, sin = c.float().cuda().contiguous(), s.float().cuda().contiguous()
        q = torch.empty(n, nh, d, dtype=dtype, device="cuda")
        K.qk_norm_rope_store(qkv.cuda(), nh, nkv, d, True, None, None, 0.0, cos, sin, rot, dev(positions), dev(req), table.cuda(),
                             k_pages, v_pages, q, interleaved=interleaved, bias=None if bias is None else bias.cuda(), value_is_key=True)
        x = qkv[:, :cols].float() + (bias if biased else 0.0)
        raw = x.view(n, nh + nkv, d)
        turn = pp.rotate_neighbours if interleaved else pp.rotate_halves
        turned = turn(raw, torch.tensor(positions), 100.0, rot) if rot else raw
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        assert rel_err(q.float(), turned[:, :nh]) < tol
        touched = torch.zeros(k_pages.shape[0], page, dtype=torch.bool)
        for i, (r, pos) in enumerate(zip(req, positions)):
            pg = int(table[r, pos // page])
            if pg < 0:
                continue
            assert rel_err(k_pages[pg, :, pos % page].float(), turned[i, nh:]) < tol
            assert rel_err(v_pages[pg, :, pos % page].float(), raw[i, nh:]) < tol
            touched[pg, pos % page] = True
            if i + 1 == n or req[i + 1] != r:              # zeros behind a request's last value
                assert bool((v_pages[pg, :, pos % page + 1:] == 0).all())
                v_pages[pg, :, pos % page + 1:] = 5.0
        untouched = ~touched.cuda()
        assert bool((k_pages.transpose(1, 2)[untouched] == 5.0).all()) and bool((v_pages.transpose(1, 2)[untouched] == 5.0).all())
    assert K.row_fault(dtype) is None


@pytest.mark.parametrize("mode", [0, 1, 2])
@pytest.mark.parametrize("n,top,groups,keep", [(6, 2, 3, 2), (9, 3, 3, 1), (1, 1, 1, 1), (5, 2, 5, 3), (64, 8, 8, 4), (256, 8, 8, 4),
                                               (12, 4, 0, 0), (7, 3, 0, 0), (40, 5, 20, 3), (600, 4, 3, 3)])
def test_grouped_choice_of_experts(n, top, groups, keep, mode):
    from inferrs_b200 import kernels as K
    g = torch.Generator().manual_seed(n + top)
    z = torch.randn(50, n + 2, generator=g) * 2
    correction = torch.randn(n, generator=g) - 0.5            # choice scores of both signs
    bias = torch.randn(n, generator=g) * 0.3
    for use_bias, use_correction, shared, scale in ((False, True, False, 1.0), (True, True, True, 2.5), (False, False, False, 0.5)):
        r = K.Router(n_experts=n, top=top, bias=bias.cuda() if use_bias else None, correction=correction.cuda() if use_correction else None,
                     has_shared=shared, groups=groups, keep=keep, mode=mode, scale=scale)
        got = torch.empty(50, r.columns, device="cuda")
        K.route(z.cuda(), r, got, torch.float32)
        want = torch.empty(50, r.columns)
        R.route(z, K.Router(**{**r.__dict__, "bias": bias if use_bias else None, "correction": correction if use_correction else None}), want)
        assert torch.equal(got.cpu() != 0, want != 0) and rel_err(got, want) < 1e-5
        if mode == 1 and use_correction and not use_bias and not shared:
            s = torch.sigmoid(z[:, :n])
            chosen = pp.chosen_experts(s, correction, top, {"count": groups, "keep": keep} if groups else None)
            assert [sorted(c) for c in chosen] == [row.nonzero().flatten().tolist() for row in got.cpu()]
    with pytest.raises(K.KernelError):
        K.route(z.cuda(), K.Router(n_experts=n, top=n + 1), torch.empty(50, n, device="cuda"), torch.float32)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,n_experts,top,groups,keep", [(96, 6, 2, 3, 2), (90, 5, 1, 0, 0), (2048, 8, 2, 4, 2), (4096, 64, 8, 8, 4),
                                                             (77, 9, 3, 3, 1), (12288, 4, 2, 2, 2), (512, 256, 8, 8, 4)])
def test_sum_norm_and_route_in_one_pass(width, n_experts, top, groups, keep, dtype):
    """Every combination of what may join the stream, with and without a choice of rows, with and without a router."""
    from inferrs_b200 import kernels as K
    g = torch.Generator().manual_seed(width)
    n, eps = 7, 1e-5
    x, plus = torch.randn(n, width, generator=g) * 3, torch.randn(n, width, generator=g)
    y, bias = torch.randn(n, width, generator=g).to(dtype), torch.randn(width, generator=g)
    weight = 1 + 0.2 * torch.randn(width, generator=g)
    router_w = (torch.randn(n_experts, width, generator=g) * 2 / width ** 0.5).to(dtype)
    correction = torch.randn(n_experts, generator=g) * 0.3
    router = K.Router(n_experts=n_experts, top=top, correction=correction.cuda(), groups=groups, keep=keep, mode=K.ROUTE_SIGMOID_SHARE,
                      scale=2.5, weight=router_w.cuda())
    assert K.sum_norm_routes(width, router)
    for delta, with_bias, with_plus in ((True, True, True), (True, False, False), (False, False, True), (True, True, False),
                                        (False, False, False)):
        total = x + (y.float() if delta else 0) + (bias if with_bias else 0) + (plus if with_plus else 0)
        want = pp.norm(total, weight, eps)
        args = (act(y, dtype) if delta else None, bias.cuda() if with_bias else None, plus.cuda() if with_plus else None)
        for chosen, routed in ((None, True), (None, False), ([5, 0, 5], False)):
            res, out = x.cuda(), torch.empty(n if chosen is None else 3, width, dtype=dtype, device="cuda")
            shares = torch.empty(n, n_experts, device="cuda") if routed else None
            K.sum_norm_route(res, *args, weight.cuda(), eps, out, rows=None if chosen is None else dev(chosen),
                             router=router if routed else None, shares=shares)
            assert rel_err(out.float(), want if chosen is None else want[chosen]) < (1e-5 if dtype == torch.float32 else 1e-2)
            assert rel_err(res, total if chosen is None else x) < 1e-6
            if routed:                 # by the row that went out: its logits in float32
                s = torch.sigmoid(out.float().cpu() @ router_w.float().T)
                ref = torch.zeros(n, n_experts)
                for t, chosen_e in enumerate(pp.chosen_experts(s, correction, top, {"count": groups, "keep": keep} if groups else None)):
                    for e in chosen_e:
                        ref[t, e] = s[t, e] / (s[t, chosen_e].sum() + 1e-20) * 2.5
                assert rel_err(shares, ref) < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("experts_n,ff", [(6, 24), (5, 33), (8, 64)])
def test_routed_gate_between_wider_rows(experts_n, ff, dtype):
    """The experts' columns inside a wider projection, their results inside a wider row."""
    from inferrs_b200 import kernels as K
    g = torch.Generator().manual_seed(ff)
    inner = experts_n * ff
    for first, extra, o_first, o_extra in ((0, 0, 0, 0), (40, 8, 24, 16), (3, 7, 5, 1)):
        wide = torch.randn(9, first + 2 * inner + extra, generator=g).to(dtype)
        shares = torch.rand(9, experts_n, generator=g) * (torch.rand(9, experts_n, generator=g) > 0.5)
        out = torch.full((9, o_first + inner + o_extra), 7.0, dtype=dtype, device="cuda")
        K.routed_gate(wide.cuda()[:, first:first + 2 * inner], shares.cuda(), experts_n, ff, out[:, o_first:o_first + inner])
        gate, up = wide[:, first:first + inner].float(), wide[:, first + inner:first + 2 * inner].float()
        want = gate * torch.sigmoid(gate) * up * shares.repeat_interleave(ff, dim=1)
        assert rel_err(out[:, o_first:o_first + inner].float(), want) < (1e-5 if dtype == torch.float32 else 1e-2)
        assert bool((out[:, :o_first] == 7.0).all()) and bool((out[:, o_first + inner:] == 7.0).all())


def test_the_embedding_rows_are_kept_for_later_passes():
    from inferrs_b200 import kernels as K
    g = torch.Generator().manual_seed(1)
    table = torch.randn(50, 90, generator=g).to(torch.bfloat16)
    ids = [3, 49, 0, 3, 17]
    out, kept = torch.empty(5, 90, device="cuda"), torch.empty(5, 90, device="cuda")
    K.embedding_gather(table.cuda(), dev(ids), out, torch.bfloat16, 12.5, copy=kept)
    assert rel_err(out, table[ids].float() * 12.5) < 1e-6 and torch.equal(out, kept)
