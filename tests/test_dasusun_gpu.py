"""The Dasusun design on the GPU against its plain statement: whole models under every cutting, batches, slots and
pages used again, replayed steps, the engine's entry points, keys at the edges of windows and far away, and every
new kernel alone."""
from __future__ import annotations

import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_dasusun as pd
from dasusun_cases import CASE_A, CASE_B, CASE_C, CASES, latent, make_weights, model, random_case
from helpers import cut, random_tokens, rel_err

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 2e-4, torch.bfloat16: 6e-2}
SEEDS = {"A": 11, "B": 12, "C": 13, "D": 14}


def assert_close(got, want, dtype):
    """float32: every row within 2e-4 of its largest value.  bfloat16: an average over depth may cancel most of what
    it adds up and amplify rounding, so the rows are judged together: their median error and the nineteenth of twenty."""
    if isinstance(got, (list, tuple)):                   # several requests: their rows are judged together
        got, want = torch.cat(list(got)), torch.cat(list(want))
    if dtype == torch.float32:
        assert rel_err(got, want) < TOL[dtype]
        return
    got, want = got.detach().double().cpu(), want.detach().double().cpu()
    assert got.shape == want.shape and bool(torch.isfinite(got).all())
    err = (got - want).abs().amax(dim=1) / want.abs().amax(dim=1).clamp_min(1e-30)
    assert float(err.median()) < 2.5e-2, float(err.median())
    assert float(torch.quantile(err, 0.95)) < TOL[dtype], float(torch.quantile(err, 0.95))


def make_runner(case, w, dtype, n_pages=24, max_requests=3, page_size=16, use_graphs=False, shapes=None):
    from inferrs_b200.engine.loading import spec_from_config
    from inferrs_b200.engine.runner import ModelRunner
    from inferrs_b200.runtime import Runtime
    spec, _ = spec_from_config(case, tensor_shapes=shapes)
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
    toks = random_tokens(75, case["vocab"], seed=3)
    want = pd.forward(case, w, toks)
    runner = make_runner(case, w, dtype)
    runner.admit("whole")
    assert_close(runner.step([entry("whole", toks)]), want, dtype)
    runner.release("whole")
    # one token a step from an empty cache: the first tokens of a sequence, and decoding through cache and state
    runner.admit("single")
    rows = [runner.step([entry("single", [t])]) for t in toks[:60]]
    assert_close(torch.cat(rows), want[:60], dtype)
    runner.release("single")
    # portions of changing size, down to two tokens and one, another request's portions beside them
    other = random_tokens(40, case["vocab"], seed=4)
    want_other = pd.forward(case, w, other)
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
    """Sizes, counts, windows, constants and the number of layers drawn from a seed: a whole prompt, then the same
    prompt in portions with its last tokens one by one, in a slot and pages that the first request has used."""
    case = random_case(seed)
    w = make_weights(case, 100 + seed)
    toks = random_tokens(90, case["vocab"], seed=seed)
    want = pd.forward(case, w, toks)
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


def test_the_stream_matches_after_every_layer():
    """What every layer hands on, through the model's own blocks, in float32: models cut off after it."""
    case, w = CASE_A, make_weights(CASE_A, 17)
    toks = random_tokens(33, case["vocab"], seed=9)
    after = []
    pd.forward(case, w, toks, after_layers=after)
    for upto in range(1, len(case["layers"]) + 1):
        short = dict(case, layers=case["layers"][:upto])
        ws = {k: v for k, v in w.items() if not k.startswith("l") or int(k[1:k.index(".")]) < upto}
        r = make_runner(short, ws, torch.float32)
        r.admit(0)
        want = pd.centred_norm(after[upto - 1], w["final.norm"], case["norm"]["eps"]) @ w["embed"].T
        assert rel_err(r.step([entry(0, toks)]), want) < TOL[torch.float32]


def test_norms_and_a_scale_of_an_absent_feed_forward():
    case = CASE_A
    w = make_weights(case, 5, bare_second=True)
    assert "l1.norm2" in w and "l1.ls2" in w and "l1.mlp.up" not in w
    toks = random_tokens(30, case["vocab"], seed=6)
    runner = make_runner(case, w, torch.float32, shapes={k: tuple(v.shape) for k, v in w.items()})
    runner.admit(0)
    assert rel_err(runner.step([entry(0, toks)]), pd.forward(case, w, toks)) < TOL[torch.float32]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_unequal_requests_in_one_batch_slots_and_pages_used_again(name, dtype):
    """Two state slots and pages for two requests; five requests of unequal length take turns, decoding side by side
    with portions of the next ones.  Every request must give what it gives alone (the plain statement knows no
    batches, slots or pages)."""
    case, w = CASES[name], make_weights(CASES[name], SEEDS[name])
    lens = {"a": 50, "b": 23, "c": 64, "d": 9, "e": 37}
    toks = {k: random_tokens(n, case["vocab"], seed=ord(k)) for k, n in lens.items()}
    want = {k: pd.forward(case, w, t) for k, t in toks.items()}
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
    assert_close([torch.cat(got[k]) for k in lens], [want[k] for k in lens], dtype)
    runner.manager.check_invariants()


@pytest.mark.parametrize("name", ["A", "B", "C", "D"])
def test_replayed_steps_give_what_plain_launches_give(name):
    """The same requests through steps captured as CUDA graphs (padding requests, the spare state slot) and through
    steps launched kernel by kernel."""
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
    want = torch.cat([pd.forward(case, w, toks["a"])[:40], pd.forward(case, w, toks["b"])[:33]])
    assert_close(outs[1][:73], want, torch.bfloat16)


def test_long_decoding_keeps_state_and_latents():
    case, w = CASE_A, make_weights(CASE_A, 21)
    toks = random_tokens(260, case["vocab"], seed=8)
    want = pd.forward(case, w, toks)
    runner = make_runner(case, w, torch.float32, n_pages=20, max_requests=1, use_graphs=True)
    runner.admit(0)
    rows = [runner.step([entry(0, toks[:5])])]
    for t in toks[5:]:
        rows.append(runner.step([entry(0, [t])]))
    assert rel_err(torch.cat(rows), want) < TOL[torch.float32]
    # the early tokens matter to the last logits: without them the far latents are other ones
    assert rel_err(pd.forward(case, w, toks[120:])[-1], want[-1]) > 1e-3


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
    n_new = 14
    want = [pd.greedy(case, w, p, n_new) for p in prompts]
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
    """A later request takes the slot and the pages of one that ended; a layer without a feed-forward brings the
    norms and the scale of one."""
    case, w = CASE_A, make_weights(CASE_A, 41, bare_second=True)
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
    wa, wb, wc = (pd.forward(case, w, toks[k]) for k in "abc")
    read = lambda s: torch.from_numpy(np.fromfile(os.path.join(out_dir, f"{s}.f32"), dtype="<f4").reshape(-1, case["vocab"]).copy())   # noqa: E731
    assert rel_err(read(0), wa[[0, 49]]) < 2e-4
    assert rel_err(read(1), torch.stack([wa[50], wb[18]])) < 2e-4
    assert rel_err(read(2), torch.stack([wb[19], wb[20], wa[69]])) < 2e-4
    assert not os.path.exists(os.path.join(out_dir, "3.f32"))
    assert rel_err(read(4), wc[[28, 29]]) < 2e-4


# ---------------------------------------------------------------------------------------------------
# keys at the edges of windows and far away, in the model: weights under which one token's value stands out
# ---------------------------------------------------------------------------------------------------
W64 = 64


def story(window, dim, rot_dim, vdim, kv_rank=64, base=10000.0):
    """One layer of two heads under whose weights a token's id is its key: the embedding is the identity times 8, the
    norms divide and do no more, the convolution adds nothing, the layer hands on its own result.  The first value of a
    head is token 9's mark, the second is the same for every token, so that the norm on the mixer's output keeps the
    share of the mark."""
    case = model(W64, W64, 1e-5, 1, [latent(2, dim, rot_dim, vdim, 64, kv_rank, 0.25, base, window)])
    w = make_weights(case, 7)
    for n in ("l0.norm1", "l0.norm1b", "final.norm"):
        w[n] = torch.zeros(W64)
    w["embed"], w["l0.canon1"], w["l0.ls1"] = torch.eye(W64) * 8.0, torch.zeros(W64, 1), torch.ones(W64)
    w["l0.dwa"] = torch.tensor([0.0, 1.0])
    w["l0.mix.dq"], w["l0.mix.dq.norm"] = torch.eye(W64), torch.ones(64)
    down = torch.zeros(kv_rank, W64)
    down[:min(kv_rank, W64)] = torch.eye(W64)[:min(kv_rank, W64)]
    w["l0.mix.dkv"], w["l0.mix.dkv.norm"] = torch.cat([down, torch.zeros(rot_dim, W64)]), torch.full((kv_rank,), (64 / kv_rank) ** 0.5)
    w["l0.mix.uq"] = torch.zeros(2 * (dim + rot_dim), 64)
    w["l0.mix.uk"] = torch.zeros(2 * dim, kv_rank)
    v = torch.zeros(vdim, kv_rank)
    v[0, 9], v[1, :] = 0.5, 0.125
    w["l0.mix.uv"] = torch.cat([v, v])
    o = torch.zeros(W64, 2 * vdim)
    o[60, 0], o[61, vdim], o[62, 1] = 1.0, 1.0, 1.0
    w["l0.mix.o"] = o
    return case, w


def run_whole_and_cut(case, w, dtype, toks, portions, single_from, single_to):
    """The logits of the whole prompt in one step, and of the same prompt in portions with the tokens
    single_from..single_to decoded one by one (a request after the whole one, in a slot and pages that it used)."""
    runner = make_runner(case, w, dtype, n_pages=60, max_requests=2)
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


def ask_for_nine(w, dim, rot_dim):
    """Head 0: token 7 asks for token 9 (channel 0 of its query and key); head 1: every token's query is the same."""
    w["l0.mix.uq"][0, 7] = 1.0
    w["l0.mix.uk"][0, 9] = 1.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window,marked_at,dim,rot_dim,vdim", [(37, 200, 32, 16, 16), (48, 208, 64, 8, 64), (5, 203, 16, 64, 8),
                                                              (64, 192, 24, 4, 24), (1, 150, 16, 2, 16), (65, 127, 8, 32, 5)])
def test_a_marked_token_is_seen_inside_the_window_and_not_beyond(window, marked_at, dim, rot_dim, vdim, dtype):
    """Token 9 stands once in a prompt of other tokens; token 7 asks for it at every distance around the window's
    edge, in a whole prompt, in portions and decoded one by one.  Its value reaches the logits while it is inside the
    window (itself and window - 1 tokens before the asking one) and not one token later."""
    case, w = story(window, dim, rot_dim, vdim)
    ask_for_nine(w, dim, rot_dim)
    n = marked_at + window + 12
    toks = [(11 + 3 * i) % 40 + 12 for i in range(n)]                 # tokens 12..51: never 7 or 9
    toks[marked_at] = 9
    asks = list(range(marked_at + max(window - 4, 1), marked_at + window + 3))
    for a in asks:
        toks[a] = 7
    want = pd.forward(case, w, toks)
    for a in asks:
        assert (float(want[a, 60]) > 0.5) == (a - marked_at < window), (a, float(want[a, 60]))
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], marked_at + max(window - 2, 1), n - 2)
    tol = 2e-4 if dtype == torch.float32 else 3e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim,rot_dim,kv_rank,marked_at", [(64, 16, 64, 15), (32, 8, 128, 16), (24, 12, 72, 255), (16, 64, 64, 0)])
def test_a_marked_token_far_back_is_found_among_hundreds(dim, rot_dim, kv_rank, marked_at, dtype):
    """Without a window: a marked token hundreds of positions back, just before and just after a page's border and at
    the very start, is found by the token that asks for it, and by no other."""
    case, w = story(None, dim, rot_dim, 16, kv_rank)
    ask_for_nine(w, dim, rot_dim)
    n = 400
    toks = [(11 + 3 * i) % 40 + 12 for i in range(n)]
    toks[marked_at] = 9
    asks = (marked_at + 1, 300, 399)
    for a in asks:
        toks[a] = 7
    want = pd.forward(case, w, toks)
    assert all(float(want[a, 60]) > 8.0 for a in asks) and float(want[298, 60]) < 2.0 and float(want[398, 60]) < 2.0
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], 290, 310)
    tol = 2e-4 if dtype == torch.float32 else 3e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("back", [0, 1, 17, 63])
def test_the_rotated_part_finds_a_token_by_its_distance(back, dtype):
    """Every token's rotated key part is the same and the queries turn it by ``back`` positions, over eight pairs of
    different speed: each token then finds the one exactly that far back, whatever stands there."""
    case, w = story(None, 8, 16, 8, base=40.0)
    rot = case["layers"][0]["mixer"]["rot"]
    base_vec = torch.cat([torch.ones(1, 1, 8), torch.zeros(1, 1, 8)], dim=-1)
    ask = pd.rotate(base_vec, torch.tensor([-back]), rot)[0, 0]
    w["l0.mix.dkv"][64:] = (base_vec[0, 0] * 0.5)[:, None].expand(16, W64)
    w["l0.mix.uq"][8:24] = (ask * 0.5)[:, None].expand(16, W64)
    case["layers"][0]["mixer"]["scale"] = 1.0
    n = 330
    toks = [(11 + 3 * i) % 40 + 12 for i in range(n)]
    for i in (3, 100, 250, 320 - back):
        toks[i] = 9
    want = pd.forward(case, w, toks)
    # (the first tokens, which have nothing that far back, take what is nearest to it)
    found = [i for i in range(back, n) if float(want[i, 60]) > 4.0]
    assert found == sorted(p + back for p in {3, 100, 250, 320 - back})
    got, got_cut = run_whole_and_cut(case, w, dtype, toks, [50, 7, 2, 64, 3], 300, 325)
    tol = 2e-4 if dtype == torch.float32 else 4e-2
    assert rel_err(got, want) < tol and rel_err(got_cut, want) < tol


# ---------------------------------------------------------------------------------------------------
# the new kernels alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,n_planes", [(96, 0), (90, 3), (512, 1), (1024, 7), (2048, 2), (4096, 5), (6144, 1), (12288, 2),
                                            (18000, 1)])
def test_post_norm_scale_average_and_norm(width, n_planes, dtype):
    """Every combination of the parts of the kernel: with and without an output to bring in, its norm, an average, the
    places where the row before and after the average goes, a choice of rows."""
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(width + n_planes)
    n, eps, post_eps = 7, 1e-5, 1e-6
    x = torch.randn(n, width, generator=g) * 30
    y = (torch.randn(n, width, generator=g) * 0.1).to(dtype)
    y[3] = 0                                                         # a row of nothing stays nothing
    post, weight = torch.randn(width, generator=g), torch.randn(width, generator=g)
    planes = torch.randn(n_planes, n, width, generator=g) * 20
    mix = torch.randn(n_planes + 1, generator=g)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    for delta, normed, average in ((True, True, True), (True, True, False), (True, False, True), (False, False, True),
                                   (False, False, False)):
        joined = x.clone()
        if delta:
            joined += pd.plain_norm(y.float(), post, post_eps) if normed else y.float()
        v = pd.depth_average(list(planes) + [joined], mix) if average else joined
        want = pd.plain_norm(v, weight, eps)
        for chosen in (None, [5, 0, 5]):
            out = torch.empty(n if chosen is None else 3, width, dtype=dtype, device="cuda")
            src, res, stream = x.cuda(), torch.zeros(n, width, device="cuda"), torch.zeros(n, width, device="cuda")
            kernels.sandwich_norm(src, y.cuda() if delta else None, post.cuda() if delta and normed else None, post_eps,
                                  weight.cuda() if normed else act(weight, torch.bfloat16), eps, out,
                                  residual=stream if chosen is None else None,
                                  planes=planes.cuda() if average and n_planes else None, mix=mix.cuda() if average else None,
                                  result=res if chosen is None else None, rows=None if chosen is None else dev(chosen))
            w = want if normed else pd.plain_norm(v, weight.to(torch.bfloat16).float(), eps)
            assert rel_err(out.float(), w if chosen is None else w[chosen]) < tol
            if chosen is None:
                assert rel_err(res, joined) < 1e-5 and rel_err(stream, v) < 1e-5
            assert torch.equal(src.cpu(), x)
    # in place, as the blocks use it
    src = x.cuda()
    out = torch.empty(n, width, dtype=dtype, device="cuda")
    kernels.sandwich_norm(src, y.cuda(), post.cuda(), post_eps, weight.cuda(), eps, out, residual=src)
    assert rel_err(src, x + pd.plain_norm(y.float(), post, post_eps)) < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width,taps", [(96, 4), (90, 2), (64, 1), (2048, 3), (4100, 5), (77, 3)])
def test_single_rows_go_through_the_convolution_in_the_norm_kernel(width, taps, dtype):
    """A portion through the kernels that convolve rows, then single rows of two requests (in changing order) through
    the norm kernel that convolves and moves the kept inputs itself, then a portion again."""
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(width + taps)
    x = [torch.randn(12, width, generator=g), torch.randn(11, width, generator=g)]
    weight, cw = torch.randn(width, generator=g), torch.randn(width, taps, generator=g)
    h = [pd.plain_norm(t, weight, 1e-5) for t in x]
    want = [t + pd.causal_conv(t, cw) for t in h]
    conv_w = cw.t().contiguous().cuda()
    state = torch.full((4, 4 + (taps - 1) * width), 0.0, device="cuda")
    state[1] = 7.0                                                    # another request's slot stays as it is
    slots, got = [3, 0], [[], []]

    def portion(a, b):
        rows = torch.cat([x[0][a[0]:a[1]], x[1][b[0]:b[1]]]).cuda()
        n0 = a[1] - a[0]
        q_start, req = dev([0, n0, rows.shape[0]]), dev([0] * n0 + [1] * (rows.shape[0] - n0))
        normed, out = (torch.empty(rows.shape, dtype=dtype, device="cuda") for _ in range(2))
        kernels.sandwich_norm(rows, None, None, 0.0, weight.cuda(), 1e-5, normed)
        kernels.causal_conv_rows(normed, 0, conv_w, state if taps > 1 else None, 4, q_start, dev(slots), req, out, True)
        kernels.conv_state_shift(normed, 0, width, taps, state, 4, q_start, dev(slots), 2)
        got[0].append(out[:n0].float().cpu())
        got[1].append(out[n0:].float().cpu())

    portion((0, 3), (0, 1))
    for i in range(5):
        order = [0, 1] if i % 2 else [1, 0]
        rows = torch.stack([x[r][(3, 1)[r] + i] for r in order]).cuda()
        out = torch.empty(rows.shape, dtype=dtype, device="cuda")
        kernels.sandwich_norm(rows, None, None, 0.0, weight.cuda(), 1e-5, out,
                              conv=(conv_w, state if taps > 1 else None, 4, dev([slots[r] for r in order]), dev([0, 1])))
        for k, r in enumerate(order):
            got[r].append(out[k:k + 1].float().cpu())
    portion((8, 12), (6, 11))
    for r in range(2):
        assert rel_err(torch.cat(got[r]), want[r]) < (1e-5 if dtype == torch.float32 else 3e-2)
    assert bool((state[1] == 7.0).all())


def rotation(rot_dim, width, at, base, positions=512, scaling=None, dims=None):
    """The package's description of a rotated part, with tables from the plain frequencies."""
    from inferrs_b200 import kernels
    rot = {"dims": rot_dim if dims is None else dims, "base": base, "scaling": scaling}
    f, factor = pd.frequencies(rot)
    ang = torch.arange(positions, dtype=torch.float64)[:, None] * f[None, :]
    return rot, kernels.LatentRotation(at=at, src=rot_dim, width=width, half=rot["dims"] // 2,
                                       cos=(torch.cos(ang) * factor).float().cuda().contiguous(),
                                       sin=(torch.sin(ang) * factor).float().cuda().contiguous())


SCALED = {"factor": 4.0, "original": 64, "fast": 8.0, "slow": 0.5}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("q_rank,kv_rank,rank,rot_dim,width,dims", [(36, 40, 64, 12, 16, 12), (64, 64, 64, 16, 16, 16),
                                                                    (17, 33, 64, 10, 16, 6), (1536, 512, 512, 64, 64, 64),
                                                                    (128, 128, 128, 2, 16, 2), (24, 72, 80, 8, 24, 0)])
def test_latents_and_the_rotated_part_are_normed_turned_and_stored(q_rank, kv_rank, rank, rot_dim, width, dims, dtype):
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(q_rank + kv_rank)
    lens, held, page = [9, 1, 20], [30, 64, 0], 16
    n = sum(lens)
    proj = torch.randn(n, 5 + q_rank + kv_rank + rot_dim + 3, generator=g).to(dtype)
    if q_rank % 8 == 0:
        proj = torch.randn(n, q_rank + kv_rank + rot_dim, generator=g).to(dtype)
    q_col = 0 if q_rank % 8 == 0 else 5
    qw, kw = 1 + 0.2 * torch.randn(q_rank, generator=g), 1 + 0.2 * torch.randn(kv_rank, generator=g)
    qw, kw = qw.to(dtype), kw.to(dtype)
    rot, described = rotation(rot_dim, width, rank, 100.0, scaling=SCALED, dims=dims)
    need = [(a + b + page - 1) // page for a, b in zip(lens, held)]
    order = torch.randperm(sum(need) + 2, generator=g).tolist()
    table = torch.full((3, max(need) + 1), -1, dtype=torch.int32)
    at = 0
    for r, k in enumerate(need):
        table[r, :k] = torch.tensor(order[at:at + k], dtype=torch.int32)
        at += k
    table[1, 64 // page] = -1                                          # a request without a page there: nothing is written
    plane = torch.full((sum(need) + 2, page, rank + width), float("nan"), dtype=dtype, device="cuda")
    positions = [h + i for h, k in zip(held, lens) for i in range(k)]
    req = [r for r, k in enumerate(lens) for _ in range(k)]
    cq = torch.empty(n, q_rank, dtype=dtype, device="cuda")
    kernels.latent_norm_store(proj.cuda(), q_col, qw.cuda(), cq, q_col + q_rank, kw.cuda(), plane, table.cuda(), dev(req),
                              dev(positions), 1e-5, rot=described)
    p = proj.float()
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    assert rel_err(cq.float(), pd.plain_norm(p[:, q_col:q_col + q_rank], qw.float(), 1e-5)) < tol
    k0 = q_col + q_rank
    c = pd.plain_norm(p[:, k0:k0 + kv_rank], kw.float(), 1e-5)
    tail = p[:, None, k0 + kv_rank:k0 + kv_rank + rot_dim]
    turned = (pd.rotate(tail, torch.tensor(positions), rot) if dims else tail)[:, 0]
    written = 0
    for i, (r, pos) in enumerate(zip(req, positions)):
        pg = int(table[r, pos // page])
        if pg < 0:
            continue
        got = plane[pg, pos % page].float().cpu()
        assert rel_err(got[:kv_rank], c[i]) < tol and rel_err(got[rank:rank + rot_dim], turned[i]) < tol
        assert bool((got[kv_rank:rank] == 0).all()) and bool((got[rank + rot_dim:] == 0).all())
        written += 1
    assert written == n - 1 and int((~torch.isnan(plane[:, :, 0].float())).sum()) == written


def scored(q_lat, q_rot, c, k_rot, scale, positions, window):
    """out[h, i] = sum_j softmax_j(scale (q_lat[h, i] . c_j + q_rot[h, i] . k_rot_j)) c_j over what position i sees."""
    s = (torch.einsum("hir,jr->hij", q_lat, c) + torch.einsum("hie,je->hij", q_rot, k_rot)) * scale
    dist = torch.as_tensor(positions)[:, None] - torch.arange(c.shape[0])[None, :]
    see = (dist >= 0) & ((dist < window) if window is not None else True)
    return torch.einsum("hij,jr->hir", pd.softmax_over_visible(s, see[None]), c)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("slices", [1, 3])
@pytest.mark.parametrize("H,R,rot_dim,width,window", [(8, 128, 16, 16, None), (3, 64, 12, 16, 23), (18, 256, 64, 64, 70),
                                                      (1, 32, 2, 16, 1), (16, 512, 64, 64, 129), (5, 50, 10, 10, 33),
                                                      (17, 96, 20, 32, 64), (2, 160, 128, 128, None)])
def test_attention_over_latents_with_a_rotated_part(H, R, rot_dim, width, window, slices, dtype):
    """Prompt portions (two tokens per block where the tensor-core form takes them), single tokens and a request at its
    first token in one step, keys in one slice and in three, against the plain sums; the queries' parts are turned
    inside the kernel."""
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(H * 100 + R)
    page, lens, held = 16, [45, 1, 1, 2], [130, 77, 0, 63]
    rot, described = rotation(rot_dim, width, R, 100.0, scaling=SCALED)
    n = sum(lens)
    scale = 1.0 / (R + rot_dim) ** 0.5
    q_lat = (torch.randn(H, n, R, generator=g) * 1.5).to(dtype)
    wide = torch.randn(n, H, 7 + rot_dim, generator=g).to(dtype)         # the rotated parts as a slice of wider heads
    plane = torch.full((40, page, R + width), float("nan"))
    table = torch.full((4, 12), -1, dtype=torch.int32)
    order = torch.randperm(40, generator=g).tolist()
    caches, positions, req = [], [], []
    for r, (a, b) in enumerate(zip(held, lens)):
        vec = torch.zeros(a + b, R + width)
        vec[:, :R + rot_dim] = torch.randn(a + b, R + rot_dim, generator=g)
        vec = vec.to(dtype).float()
        caches.append(vec)
        for p in range((a + b + page - 1) // page):
            table[r, p] = order.pop()
            part = vec[p * page:(p + 1) * page]
            plane[table[r, p], :part.shape[0]] = part
        positions += range(a, a + b)
        req += [r] * b
    out = torch.empty(H, n, R, dtype=dtype, device="cuda")
    q_start = [0] + list(np.cumsum(lens))
    tiles = None
    if slices == 1:
        tile = [(-1, 0)] + [(r, q_start[r] + i) for r in range(4) for i in range(0, lens[r], kernels.LATENT_TILE_TOKENS)]
        tiles = (dev([t[0] for t in tile]), dev([t[1] for t in tile]), len(tile), dev([int(v) for v in q_start]))
    kernels.latent_attention(q_lat.cuda(), act(plane, dtype), table.cuda(), dev(req), dev(positions), scale, window, out, slices,
                             tiles, q_rot=wide.cuda()[:, :, 7:], rot=described)
    q_rot = pd.rotate(wide.float()[:, :, 7:], torch.tensor(positions), rot).transpose(0, 1)
    for r in range(4):
        rows = slice(int(q_start[r]), int(q_start[r + 1]))
        want = scored(q_lat.float()[:, rows], q_rot[:, rows], caches[r][:, :R], caches[r][:, R:R + rot_dim], scale,
                      positions[rows], window)
        assert rel_err(out[:, rows].float(), want) < (2e-5 if dtype == torch.float32 else 2e-2), r


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("slices", [1, 4])
def test_attention_over_latents_sees_exactly_its_keys_by_the_rotated_part(slices, dtype):
    """The rotated part of one cached vector is made to stand out, so that whoever sees it gives its latent: just inside
    and just outside the window, at borders of pages and of key tiles, at the first token."""
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(4)
    R, P, H, page, T = 64, 16, 3, 16, 300
    rot, described = rotation(P, 16, R, 100.0)
    c = torch.randn(T, R, generator=g).to(dtype)
    for j, pos, window in ((0, 0, None), (0, 299, None), (63, 250, None), (64, 250, None), (255, 255, 1), (254, 255, 1),
                           (200, 263, 64), (199, 263, 64), (16, 100, 85), (15, 100, 85), (127, 191, 65), (126, 191, 65)):
        k_rot = torch.zeros(1, 1, P)
        k_rot[0, 0, 0], k_rot[0, 0, 1] = 4.0, 4.0
        plane_vec = torch.zeros(T, R + P)
        plane_vec[:, :R] = c.float()
        plane_vec[j, R:] = pd.rotate(k_rot, torch.tensor([j]), rot)[0, 0]
        # a query that, turned by its own position, meets the key turned by j: the score is large there and zero elsewhere
        q_rot = pd.rotate(k_rot, torch.tensor([j - pos]), rot).expand(1, H, P).contiguous().to(dtype)
        plane = torch.full((25, page, R + P), float("nan"))
        order = torch.randperm(25, generator=g).tolist()
        table = torch.tensor([order[:(T + page - 1) // page]], dtype=torch.int32)
        for p in range(table.shape[1]):
            part = plane_vec[p * page:(p + 1) * page]
            plane[order[p], :part.shape[0]] = part
        out = torch.empty(H, 1, R, dtype=dtype, device="cuda")
        kernels.latent_attention(torch.zeros(H, 1, R, dtype=dtype, device="cuda"), act(plane, dtype), table.cuda(), dev([0]),
                                 dev([pos]), 1.0, window, out, slices, q_rot=q_rot.cuda(), rot=described)
        seen = j <= pos and (window is None or pos - j < window)
        got = out[:, 0].float().cpu()
        lo = 0 if window is None else max(0, pos - window + 1)
        want = c[j].float() if seen else c[lo:pos + 1].float().mean(0)
        assert rel_err(got, want.expand(H, R)) < (1e-5 if dtype == torch.float32 else 3e-2), (j, pos, window)


@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_products_read_and_write_slices_of_heads(dtype):
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(6)
    for n, H, K, P, M in ((21, 5, 24, 12, 40), (1, 3, 7, 3, 9), (64, 16, 64, 32, 128), (33, 2, 64, 16, 512)):
        x = torch.randn(n, H, K + P, generator=g).to(dtype)
        w = (torch.randn(H, M, K, generator=g) / K ** 0.5).to(dtype)
        out = torch.empty((n, H * M), dtype=dtype, device="cuda")
        kernels.batched_linear(x.cuda()[:, :, :K].transpose(0, 1), w.cuda(), out.view(n, H, M).transpose(0, 1), dtype)
        want = torch.einsum("nhk,hmk->nhm", x.float()[:, :, :K], w.float()).reshape(n, H * M)
        assert rel_err(out.float(), want) < (1e-5 if dtype == torch.float32 else 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,k,inner", [(1, 96, 72), (5, 64, 136), (16, 128, 1024), (16, 2048, 256), (17, 90, 33), (3, 45, 50),
                                          (200, 160, 264), (8, 8192, 128)])
def test_gelu_behind_a_product(rows, k, inner, dtype):
    """A few rows (the product takes gelu itself, with and without its K range cut over a cluster) and many (a kernel
    after the product)."""
    from inferrs_b200 import kernels
    g = torch.Generator().manual_seed(rows * 7 + inner)
    x, w = torch.randn(rows, k, generator=g).to(dtype), (torch.randn(inner, k, generator=g) * (2.0 / k ** 0.5)).to(dtype)
    out = torch.empty(rows, inner, dtype=dtype, device="cuda")
    kernels.gelu_linear(x.cuda(), w.cuda(), out, dtype)
    assert rel_err(out.float(), pd.gelu_tanh(x.float() @ w.float().T)) < (2e-5 if dtype == torch.float32 else 2e-2)
    if dtype == torch.bfloat16 and k % 8 == 0:
        for split in (1, 2, 4):
            if k // 64 >= split:
                kernels.gemm_tn_tcgen05(x.cuda(), w.cuda(), out, split_k=split, gelu=True)
                assert rel_err(out.float(), pd.gelu_tanh(x.float() @ w.float().T)) < 2e-2
        assert kernels.gemm_tcgen05_error() == 0
