"""The Gedilorn decoder in the engine against the plain implementation (needs a GPU): whole prompts, token-by-token
decoding, portions, ragged batches, slots and pages used again, long decoding, generation through the public entry point and
the command line, the replay program.  The kernels alone are in test_gedilorn_kernels_gpu.py."""
import json
import math
import os
import subprocess

import numpy as np
import pytest
import torch

from helpers import GEDILORN_CONFIGS, ROOT, TraceRun, random_tokens
from plain import gedilorn_plain as P

pytestmark = pytest.mark.gpu

TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
NAMES = ["GA", "GB", "GC", "GD", "GE", "GF"]
_models, _plains, _refs = {}, {}, {}


def engine(folders, name, dtype):
    import rocmforge_b200 as rf
    if (name, dtype) not in _models:
        _models[(name, dtype)] = rf.Model.from_folder(folders(name, dtype), dtype=TORCH[dtype])
    return _models[(name, dtype)]


def plain_model(folders, name, dtype):
    from safetensors.torch import load_file
    if (name, dtype) not in _plains:
        folder = folders(name, dtype)
        _plains[(name, dtype)] = P.PlainGedilorn(json.load(open(os.path.join(folder, "config.json"))),
                                                load_file(os.path.join(folder, "model.safetensors")))
    return _plains[(name, dtype)]


def plain_logits(folders, name, dtype, tokens):
    """Logits of the plain model on the folder's stored (rounded) weights, every position."""
    key = (name, dtype, tuple(tokens))
    if key not in _refs:
        _refs[key] = plain_model(folders, name, dtype).logits(list(tokens))
    return _refs[key]


def row_errors(got, ref):
    """Per row: root mean square of the difference (mean taken off) over the root mean square of the reference logits."""
    got = torch.as_tensor(np.asarray(got), dtype=torch.float64)
    ref = torch.as_tensor(np.asarray(ref), dtype=torch.float64)
    assert got.shape == ref.shape and torch.isfinite(got).all()
    d = got - ref
    d = d - d.mean(dim=-1, keepdim=True)
    return d.pow(2).mean(dim=-1).sqrt() / (ref - ref.mean(dim=-1, keepdim=True)).pow(2).mean().sqrt()


def close(got, ref, dtype, what):
    """Rows compared by the root mean square of their difference as a share of the logits' spread: 32-bit within 3e-4 (the
    sums' order differs from the float64 model's), bfloat16 2 % on average and none beyond 8 %."""
    err = row_errors(got, ref)
    if dtype == "float32":
        assert float(err.max()) < 3e-4, f"{what}: row errors up to {float(err.max()):.2e} (row {int(err.argmax())})"
        return
    assert float(err.mean()) < 0.02 and float(err.max()) < 0.08, \
        f"{what}: row errors up to {float(err.max()):.3f} (row {int(err.argmax())}), mean {float(err.mean()):.3f}"


def vocab(name):
    return GEDILORN_CONFIGS[name]["vocab"]


def poison_free_pages(cache):
    for g in cache.groups:
        free = [p for p in range(g.n_pages) if not g.pool.is_held(p)]
        if free:
            idx = torch.tensor(free, device=g.storage.device)
            g.storage[:, :, idx] = float("nan")
            if g.value_storage is not None:
                g.value_storage[:, :, idx] = float("nan")


# --------------------------------------------------------------------------- the model in the engine

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_whole_prompt(folders, name, dtype):
    """Every position of a prompt that crosses four page borders."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    toks = random_tokens(vocab(name), 270, 3)
    cache = m.new_cache(max_tokens=512, max_slots=2)
    poison_free_pages(cache)
    s = cache.alloc_slot()
    got = m.step(cache, [StepRequest(s, toks, range(len(toks)))]).cpu()
    close(got, plain_logits(folders, name, dtype, toks), dtype, f"{name} {dtype} whole prompt")


@pytest.mark.parametrize("name", NAMES)
def test_the_stream_after_every_layer(folders, name, monkeypatch):
    """The 32-bit residual stream after each layer against the plain model's, so that a fault names its layer."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, "float32")
    toks = random_tokens(vocab(name), 90, 4)
    want = []
    plain_model(folders, name, "float32").logits(toks, trace=want)
    cache = m.new_cache(max_tokens=256, max_slots=1)
    s = cache.alloc_slot()
    got = []
    for block in m.spec.blocks:
        def recording(ctx, stream, view, inner=block.forward):
            inner(ctx, stream, view)
            stream.flush()
            h = stream.h.detach()
            got.append((h.sum(dim=1) if h.dim() == 3 else h).cpu().clone())
        monkeypatch.setattr(block, "forward", recording)
    m.step(cache, [StepRequest(s, toks, range(len(toks)))])
    assert len(got) == len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        assert float((g.double() - w).abs().max()) < 2e-5 * max(1.0, float(w.abs().max())), f"{name}: the stream differs after layer {i}"


@pytest.mark.parametrize("name", ["GA", "GC", "GD"])
def test_token_by_token_from_the_first_token(folders, name):
    """One token a step from an empty cache: the first token (which has no token before it), page borders; and the same
    logits as the prompt in one step."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, "float32")
    toks = random_tokens(vocab(name), 150, 5)
    ref = plain_logits(folders, name, "float32", toks)
    cache = m.new_cache(max_tokens=512, max_slots=2)
    s = cache.alloc_slot()
    got = torch.cat([m.step(cache, [StepRequest(s, [t], [0])]).cpu() for t in toks])
    close(got, ref, "float32", f"{name} token by token")
    s2 = cache.alloc_slot()
    whole = m.step(cache, [StepRequest(s2, toks, range(len(toks)))]).cpu()
    assert float(row_errors(got, whole).max()) < 1e-4


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_portions_of_many_sizes(folders, name, dtype):
    """A prompt cut into portions of 1 to 70 tokens (some worked on like single tokens, some that gather their context again):
    a portion's first token finds the token before it after portions of odd and even length; positions count from the
    sequence's start, not a portion's."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    sizes = [2, 3, 64, 1, 5, 17, 2, 70, 33, 2, 1, 8, 40]
    toks = random_tokens(vocab(name), sum(sizes), 7)
    cache = m.new_cache(max_tokens=512, max_slots=2)
    poison_free_pages(cache)
    s = cache.alloc_slot()
    got, at = [], 0
    for n in sizes:
        got.append(m.step(cache, [StepRequest(s, toks[at:at + n], range(n))]).cpu())
        at += n
    close(torch.cat(got), plain_logits(folders, name, dtype, toks), dtype, f"{name} {dtype} portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_ragged_batch_then_decoding_with_slots_used_again(folders, name, dtype):
    """Unequal prompts in one step (one of a single token), decoded together; requests end at different steps, their slots
    (each with its last token) and pages go to new requests; every request must equal the plain model's logits for it alone."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    V = vocab(name)
    lens = [(1, 30), (70, 12), (131, 25), (2, 6)]
    seqs = [random_tokens(V, a + b, 20 + i) for i, (a, b) in enumerate(lens)]
    refs = [plain_logits(folders, name, dtype, t) for t in seqs]
    cache = m.new_cache(max_tokens=64 * 8, max_slots=4)
    poison_free_pages(cache)
    slots = [cache.alloc_slot() for _ in lens]
    got = m.step(cache, [StepRequest(sl, t[:a], [0, a - 1]) for sl, t, (a, _) in zip(slots, seqs, lens)]).cpu()
    want = torch.stack([r[i] for r, (a, _) in zip(refs, lens) for i in (0, a - 1)])
    close(got, want, dtype, f"{name} {dtype} ragged prompts")
    live = list(range(len(lens)))
    for step in range(30):
        for i in [i for i in live if lens[i][1] <= step]:
            cache.free_slot(slots[i]); live.remove(i)
        poison_free_pages(cache)
        got = m.step(cache, [StepRequest(slots[i], [seqs[i][lens[i][0] + step]], [0]) for i in live]).cpu()
        close(got, torch.stack([refs[i][lens[i][0] + step] for i in live]), dtype, f"{name} {dtype} batch decode step {step}")
    for i in live:
        cache.free_slot(slots[i])
    # the freed slots again: a last token that was taken for the new request's own, or a page that kept old rows, would show
    again = [random_tokens(V, n, 40 + n) for n in (45, 9)]
    slots = [cache.alloc_slot() for _ in again]
    got = m.step(cache, [StepRequest(sl, t, [0, len(t) - 1]) for sl, t in zip(slots, again)]).cpu()
    want = torch.cat([plain_logits(folders, name, dtype, t)[[0, len(t) - 1]] for t in again])
    close(got, want, dtype, f"{name} {dtype} reused slots")


def test_a_batch_changes_nothing_beyond_rounding(folders):
    """A request's logits in a batch of unequal requests equal its logits alone up to the order of 32-bit sums (products of
    few tokens cut K into partial sums, products of many do not), in the prompt step and in decoding."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, "GB", "float32")
    V = vocab("GB")
    seqs = [random_tokens(V, n, 80 + n) for n in (150, 3, 77)]
    cache = m.new_cache(max_tokens=64 * 12, max_slots=6)
    alone_rows = []
    for t in seqs:
        s = cache.alloc_slot()
        a = [m.step(cache, [StepRequest(s, t[:-2], [len(t) - 3])]).cpu()]
        a += [m.step(cache, [StepRequest(s, [x], [0])]).cpu() for x in t[-2:]]
        alone_rows.append(torch.cat(a))
        cache.free_slot(s)
    slots = [cache.alloc_slot() for _ in seqs]
    tog = [m.step(cache, [StepRequest(sl, t[:-2], [len(t) - 3]) for sl, t in zip(slots, seqs)]).cpu()]
    tog += [m.step(cache, [StepRequest(sl, [t[k]], [0]) for sl, t in zip(slots, seqs)]).cpu() for k in (-2, -1)]
    for i in range(len(seqs)):
        assert float(row_errors(torch.stack([x[i] for x in tog]), alone_rows[i]).max()) < 1e-4, f"request {i} depends on its batch"


@pytest.mark.parametrize("name,dtype", [("GA", "float32"), ("GC", "float32"), ("GC", "bfloat16"), ("GE", "bfloat16")])
def test_long_decoding(folders, name, dtype):
    """Three hundred single-token steps after a short prompt, two sequences side by side: five page borders, attention that
    reaches back to the first token."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    a, b = random_tokens(vocab(name), 330, 9), random_tokens(vocab(name), 330, 10)
    cache = m.new_cache(max_tokens=64 * 13, max_slots=2)
    sa, sb = cache.alloc_slot(), cache.alloc_slot()
    got = [m.step(cache, [StepRequest(sa, a[:30], [29]), StepRequest(sb, b[:30], [29])]).cpu()]
    for x, y in zip(a[30:], b[30:]):
        poison_free_pages(cache)
        got.append(m.step(cache, [StepRequest(sa, [x], [0]), StepRequest(sb, [y], [0])]).cpu())
    got = torch.stack(got)
    close(got[:, 0], plain_logits(folders, name, dtype, a)[29:], dtype, f"{name} long decoding, first sequence")
    close(got[:, 1], plain_logits(folders, name, dtype, b)[29:], dtype, f"{name} long decoding, second sequence")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_public_entry_point(folders, dtype):
    """LLM.generate: the scheduler admits unequal prompts, decode steps replay from graphs and run one
    step ahead of the host (the last token kept per sequence must survive a step that is run again), requests end at different lengths."""
    import rocmforge_b200 as rf
    name = "GC"
    llm = rf.LLM(folders(name, dtype), dtype=dtype)
    prompts = [random_tokens(vocab(name), n, 60 + n) for n in (3, 140, 11)]
    out = llm.generate(prompts, max_tokens=12, temperature=0.0, stop_token_ids=[])
    for p, r in zip(prompts, out):
        assert len(r.tokens) == 12
        seq = list(p)
        for k, tok in enumerate(r.tokens):
            row = plain_logits(folders, name, dtype, seq)[-1]
            best = int(torch.argmax(row))
            slack = (1e-5 if dtype == "float32" else 2e-2) * float(row.abs().max())
            assert tok == best or float(row[best] - row[tok]) <= slack, \
                f"request of {len(p)} tokens, generated token {k}: {tok}, plain {best}"
            seq.append(tok)


def test_command_line(folders):
    """bin/rocmforge on a Gedilorn folder: greedy tokens equal the plain model's."""
    folder = folders("GA", "float32")
    prompt = random_tokens(vocab("GA"), 9, 91)
    out = subprocess.run([os.path.join(ROOT, "bin", "rocmforge"), "--model", folder, "--dtype", "float32", "--prompt-ids",
                          ",".join(map(str, prompt)), "--max-tokens", "5", "--temperature", "0", "--stop-ids", "", "--debug"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    ids = [int(l.split("token_id=")[1]) for l in out.stderr.splitlines() if l.startswith("[Generated]")]
    seq = list(prompt)
    for tok in ids:
        row = plain_logits(folders, "GA", "float32", seq)[-1]
        assert tok == int(torch.argmax(row)) or float(row.max() - row[tok]) <= 1e-5 * float(row.abs().max())
        seq.append(tok)
    assert len(ids) == 5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program(folders, tmp_path, dtype):
    """bin/trace_run on a Gedilorn folder: whole prompts, a prompt and its last tokens one by one, and a batch."""
    name = "GC"
    V = vocab(name)
    a, b, c = random_tokens(V, 180, 71), random_tokens(V, 37, 72), random_tokens(V, 5, 73)
    ra, rb, rc = (plain_logits(folders, name, dtype, t) for t in (a, b, c))
    tr = TraceRun(folders(name, dtype), dtype, str(tmp_path / "out"), max_tokens=512)
    got = tr.step([("a", a, [0, 6, 7, 99, 100, 179])], end=["a"])
    close(got, ra[[0, 6, 7, 99, 100, 179]], dtype, "replay: whole")
    got = tr.step([("b", b[:30], [29])])
    close(got, rb[[29]], dtype, "replay: prompt")
    for i in range(30, 37):
        got = tr.step([("b", [b[i]], [0])], end=["b"] if i == 36 else [])
        close(got, rb[[i]], dtype, f"replay: decoded {i}")
    got = tr.step([("x", a[:160], [159]), ("y", c[:3], []), ("z", b[:20], [0, 19])])
    close(got, torch.stack([ra[159], rb[0], rb[19]]), dtype, "replay: batch")
    got = tr.step([("x", [a[160]], [0]), ("y", [c[3]], [0]), ("z", [b[20]], [0])], end=["y"])
    close(got, torch.stack([ra[160], rc[3], rb[20]]), dtype, "replay: batch decoded")
    assert tr.step([("x", [a[161]], []), ("z", [b[21]], [])], end=["x", "z"]) is None
    assert tr.close() == 0


def test_a_step_that_ran_ahead_and_was_dropped_changes_nothing(folders):
    """The decode runner launches the next step before the host has seen this one's ids.  A caller that goes on with another token
    than the sampled one makes it drop that step; the step it then runs must find the token before it, not the dropped one."""
    from rocmforge_b200 import SamplingParams, StepRequest
    from rocmforge_b200.engine.graph import DecodeRunner
    name = "GA"
    m = engine(folders, name, "float32")
    toks = random_tokens(vocab(name), 40, 12)
    cache = m.new_cache(max_tokens=256, max_slots=2)
    assert cache.steps_repeatable
    s = cache.alloc_slot()
    m.step(cache, [StepRequest(s, toks[:9], [])])
    runner = DecodeRunner(m, cache)
    greedy = SamplingParams(temperature=0.0)
    for k, t in enumerate(toks[9:]):
        got = runner.step_ids([s], [t], greedy, [0], [k], more=True)[0]
        row = plain_logits(folders, name, "float32", toks)[9 + k]
        assert got == int(row.argmax()) or float(row.max() - row[got]) <= 1e-5 * float(row.abs().max()), f"step {k}"
    assert runner.discarded > 20 and runner.launched_ahead >= 0
