"""The Migosun design in the engine against its plain restatement: whole prompts, prompts followed by single
tokens, portions of many sizes, unequal batches, caches so small that slots, pages and state rows are used again,
long decoding past chunk edges and page borders, greedy generation through the entry point, and the replay program."""
import functools
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_migosun as plain
from gpu_util import Recorder, run_steps, steps_batches, steps_tail, steps_whole
from tiny import repo_root
from migosun_cases import case

from esp_b200.engine import Engine, StepEntry
from esp_b200.weights import write_safetensors

pytestmark = pytest.mark.gpu

# root mean square of (engine - plain) over a row of logits, mean taken off, over the root mean square of the
# request's plain logits.  float32: only the order of sums differs.  bfloat16: activations and cached rows are
# rounded to 8 bits a few times per layer; the recurrences themselves stay 32-bit.
BOUND = {"float32": 2e-5, "bfloat16": 4e-2}


@functools.lru_cache(maxsize=None)
def model(name, seed=7):
    raw, ranks = case(name)
    return raw, plain.random_weights(raw, seed, *ranks)


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name in ("A", "B", "C"):
        raw, w = model(name)
        d = tmp_path_factory.mktemp(f"migosun_{name}")
        (d / "config.json").write_text(json.dumps(raw))
        write_safetensors(d / "model.safetensors", w)
        out[name] = d
    return out


_engines = {}


def engine_for(folder, dtype, max_tokens=2048, **kw):
    key = (str(folder), dtype, max_tokens, tuple(sorted(kw.items())))
    if key not in _engines:
        _engines[key] = Engine.from_folder(folder, dtype=dtype, max_tokens=max_tokens, **kw)
    return _engines[key]


@functools.lru_cache(maxsize=None)
def plain_logits(name, toks):
    raw, w = model(name)
    return plain.forward(raw, w, list(toks)).numpy()


@functools.lru_cache(maxsize=None)
def moved_by_rounded_norms(name, toks):
    """Per position: how far the plain logits move (in the units of BOUND) when the restatement rounds the results of its
    norms to bfloat16 and nothing else.  Random weights make some positions ill conditioned: a rounding of 2^-9 of a
    layer's input comes out a hundred times larger behind a head's norm over a nearly cancelled read-out."""
    raw, w = model(name)
    ref = plain_logits(name, toks)
    with plain.norms_rounded_to(torch.bfloat16):
        got = plain.forward(raw, w, list(toks)).numpy()
    d = got - ref
    d = d - d.mean(1, keepdims=True)
    return np.sqrt((d ** 2).mean(1)) / np.sqrt((ref ** 2).mean())




@functools.lru_cache(maxsize=None)
def moved_by_rounded_weights(name, toks):
    """The same for the restatement with all its weights moved by up to one part in 2^9, the most of three draws: where a
    rounding anywhere else (of an attention's result, say) is felt as much as one of the norms."""
    raw, w = model(name)
    ref, most = plain_logits(name, toks), 0.0
    for seed in range(3):
        g = torch.Generator().manual_seed(seed)
        moved = {n: t.double() * (1 + (torch.rand(t.shape, generator=g) - 0.5) * 2.0 ** -8) for n, t in w.items()}
        d = plain.forward(raw, moved, list(toks)).numpy() - ref
        d = d - d.mean(1, keepdims=True)
        most = np.maximum(most, np.sqrt((d ** 2).mean(1)) / np.sqrt((ref ** 2).mean()))
    return most


def requests_for(name, lengths, seed=3):
    rng = np.random.default_rng(seed)
    vocab = model(name)[0]["vocab"]
    return {f"r{i}": [int(t) for t in rng.integers(0, vocab, n)] for i, n in enumerate(lengths)}


def check(name, dtype, requests, rec, what, positions=None):
    for rid, toks in requests.items():
        ref = plain_logits(name, tuple(toks))
        at = list(range(len(toks))) if positions is None else list(positions[rid])
        got = rec.logits_of(rid, at)
        d = got - ref[at]
        d = d - d.mean(1, keepdims=True)
        err = np.sqrt((d ** 2).mean(1)) / np.sqrt((ref ** 2).mean())
        bound = np.full(len(at), BOUND[dtype])
        if dtype == "bfloat16":
            # the engine rounds at the norms and at a few more places: an ill-conditioned position may move twice as far
            # as the restatement does under its rounded norms; at most positions this adds less than 2e-2
            bound = bound + 2 * moved_by_rounded_norms(name, tuple(toks))[at]
            if (err > bound).any():
                bound = np.maximum(bound, 2 * moved_by_rounded_weights(name, tuple(toks))[at])
        worst = int(np.argmax(err / bound))
        assert err[worst] <= bound[worst], (f"{what}, case {name}, {dtype}, request {rid} ({len(toks)} tokens): position "
                                            f"{at[worst]} is off by {err[worst]:.3e} (bound {bound[worst]:.1e}); first "
                                            f"position over its bound: {at[int(np.argmax(err > bound))]}")


def steps_portions(requests, sizes):
    """Each request alone, cut into portions whose sizes cycle through ``sizes``."""
    steps = []
    for rid, toks in requests.items():
        at, i = 0, 0
        while at < len(toks):
            n = min(sizes[i % len(sizes)], len(toks) - at)
            steps.append(([(rid, toks[at:at + n], list(range(n)))], [rid] if at + n == len(toks) else []))
            at += n
            i += 1
    return steps


LENGTHS = {"A": (1, 9, 83, 150), "B": (2, 40, 77, 131), "C": (3, 64, 129, 200)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_whole_prompts(folders, name, dtype):
    reqs = requests_for(name, LENGTHS[name])
    eng = engine_for(folders[name], dtype)
    rec = Recorder(model(name)[0]["vocab"])
    run_steps(eng, steps_whole(reqs), rec)
    check(name, dtype, reqs, rec, "whole prompts")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_prefill_then_token_by_token(folders, name, dtype):
    """The last 80 tokens one by one: they pass chunk edges at multiples of 37, 64, 70 and 128, page borders at 64 and
    128, and the chunk of one position; the first requests are decoded from their second token on."""
    reqs = requests_for(name, LENGTHS[name])
    eng = engine_for(folders[name], dtype)
    rec = Recorder(model(name)[0]["vocab"])
    run_steps(eng, steps_tail(reqs, tail=80), rec)
    check(name, dtype, reqs, rec, "prompt, then single tokens")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_portions_of_many_sizes(folders, name, dtype):
    reqs = requests_for(name, LENGTHS[name][1:], seed=5)
    eng = engine_for(folders[name], dtype)
    rec = Recorder(model(name)[0]["vocab"])
    run_steps(eng, steps_portions(reqs, [2, 31, 3, 64, 17, 2, 2]), rec)
    check(name, dtype, reqs, rec, "portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_unequal_batches_in_a_cache_that_is_used_again(folders, name, dtype):
    """Two batches, one after the other, in a cache that holds one of them: every slot, page and state row of the
    second batch was used by the first.  A state that is not cleared, or a page table that keeps an old page, shows."""
    lengths = (70, 5, 140, 33, 129, 64, 2, 100)
    reqs = requests_for(name, lengths, seed=9)
    ids = list(reqs)
    batches = [ids[:4], ids[4:]]
    prompt = {rid: max(1, len(reqs[rid]) - 40 + 7 * i) for i, rid in enumerate(ids)}
    prompt = {rid: min(n, len(reqs[rid])) for rid, n in prompt.items()}
    eng = engine_for(folders[name], dtype, max_tokens=7 * 64, max_slots=4)
    rec = Recorder(model(name)[0]["vocab"])
    run_steps(eng, steps_batches(reqs, batches, prompt), rec)
    check(name, dtype, reqs, rec, "unequal batches")
    assert eng.cache.book.slots.available == 4
    assert all(g.pool.available == g.pool.n for g in eng.cache.book.groups)


@pytest.mark.parametrize("name", ["A", "B", "C"])
def test_cuttings_agree_bit_for_bit_in_float32(folders, name):
    """No sum's order depends on how a sequence is cut or what it is batched with; decode steps replay captured graphs."""
    reqs = requests_for(name, (3, 90, 150), seed=13)
    eng = engine_for(folders[name], "float32")
    outs = []
    ids = list(reqs)
    for steps in (steps_whole(reqs), steps_tail(reqs, tail=40), steps_portions(reqs, [2, 5, 64]),
                  steps_batches(reqs, [ids], {rid: max(1, len(t) - 30) for rid, t in reqs.items()})):
        rec = Recorder(model(name)[0]["vocab"])
        run_steps(eng, steps, rec)
        outs.append(rec)
    assert eng.graph_replays > 0
    for rid, toks in reqs.items():
        at = list(range(len(toks)))
        first = outs[0].logits_of(rid, at)
        for other in outs[1:]:
            assert np.array_equal(first, other.logits_of(rid, at))


def test_long_decoding_in_a_small_cache(folders):
    """300 single tokens after a prompt of 3 in a cache of 3 pages, less than the sequence: the chunked layers give
    the pages of a finished chunk back and get them again; the recurrent states carry everything older."""
    name = "A"
    reqs = requests_for(name, (303,), seed=21)
    for dtype in ("float32", "bfloat16"):
        eng = engine_for(folders[name], dtype, max_tokens=3 * 64)
        rec = Recorder(model(name)[0]["vocab"])
        run_steps(eng, steps_tail(reqs, tail=300), rec)
        check(name, dtype, reqs, rec, "long decoding")


def test_residual_stream_behind_every_layer(folders):
    name = "A"
    raw, w = model(name)
    toks = requests_for(name, (45,), seed=2)["r0"]
    layers = []
    plain.forward(raw, w, toks, trace=layers)
    eng = engine_for(folders[name], "float32")
    slot = eng.open()
    aux = {"residual_trace": []}
    eng.step([StepEntry(slot, toks, [0])], aux)
    eng.close(slot)
    assert len(aux["residual_trace"]) == len(layers)
    for i, (got, want) in enumerate(zip(aux["residual_trace"], layers)):
        err = float((got.cpu().double() - want).abs().max() / want.abs().max())
        assert err < 1e-5, f"layer {i}: {err:.2e}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_entry_point(folders, dtype):
    from esp_b200.provider import DecoderProvider, GenerationRequest
    name = "B"
    raw, w = model(name)
    prompts = list(requests_for(name, (4, 19, 70), seed=31).values())
    prov = DecoderProvider.load(folders[name], dtype=dtype, max_batch=2, max_tokens=1024)
    outs = prov.generate([GenerationRequest(prompt_ids=p, max_tokens=12) for p in prompts])
    for p, out in zip(prompts, outs):
        assert len(out.token_ids) == 12 and out.finish_reason == "length"
        # every token the engine chose is, for the plain restatement given the same prefix, the best token or
        # within rounding of it
        seq = list(p)
        for tok in out.token_ids:
            ref = plain.forward(raw, w, seq)[-1]
            slack = (1e-4 if dtype == "float32" else 0.12) * float(ref.abs().max())
            assert float(ref.max() - ref[tok]) <= slack
            seq.append(tok)


def test_the_command_line_generates(folders):
    env = dict(os.environ)
    proc = subprocess.run([sys.executable, "-m", "esp_b200", "generate", "--model", str(folders["A"]), "--dtype", "float32",
                           "--prompt-ids", "5,17,3", "--prompt-ids", "9 8 7 6 5 4", "--max-tokens", "5"],
                          capture_output=True, text=True, env=env, cwd=str(repo_root()), timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    lines = [json.loads(l) for l in proc.stdout.splitlines() if l.startswith("{")]
    assert [len(l["token_ids"]) for l in lines] == [5, 5]
    raw, w = model("A")
    want, margins = plain.greedy(raw, w, [5, 17, 3], 5)
    if min(margins) > 1e-3:
        assert lines[0]["token_ids"] == want


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program(folders, tmp_path, dtype):
    name = "A"
    reqs = requests_for(name, (1, 60, 141), seed=17)
    ids = list(reqs)
    steps = steps_tail(reqs, tail=20) + steps_batches({k + "x": v for k, v in reqs.items()}, [[i + "x" for i in ids]],
                                                      {i + "x": max(1, len(reqs[i]) - 9) for i in ids})
    lines, wanted = [], []
    for i, (entries, end) in enumerate(steps):
        lines.append(json.dumps({"step": i, "entries": [{"id": rid, "tokens": t, "want": wnt} for rid, t, wnt in entries],
                                 "end": end}))
        wanted.append(sum(len(wnt) for _, _, wnt in entries))
    proc = subprocess.run([sys.executable, str(repo_root() / "bin" / "trace_run"), "--model", str(folders[name]), "--dtype",
                           dtype, "--out", str(tmp_path), "--max-tokens", "404"], input="\n".join(lines) + "\n",
                          capture_output=True, text=True, timeout=600)
    assert proc.returncode == 0, proc.stderr[-3000:]
    assert proc.stdout.split("\n")[:len(steps)] == [f"done {i}" for i in range(len(steps))]
    vocab = model(name)[0]["vocab"]
    rec = Recorder(vocab)
    pos = {}
    for i, (entries, _end) in enumerate(steps):
        data = np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(wanted[i], vocab)
        r = 0
        for rid, toks, want in entries:
            for wnt in want:
                rec.logits.setdefault(rid, {})[pos.get(rid, 0) + wnt] = data[r]
                r += 1
            pos[rid] = pos.get(rid, 0) + len(toks)
    check(name, dtype, reqs, rec, "replay program, alone")
    rec.logits = {rid[:-1]: rows for rid, rows in rec.logits.items() if rid.endswith("x")}
    check(name, dtype, reqs, rec, "replay program, batched")
