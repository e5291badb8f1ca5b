"""The Dubodra decoder in the engine against the plain implementation (needs a GPU): whole prompts, token-by-token
decoding, portions, ragged batches, slots and pages used again, long decoding, generation through the public entry point and
the command line, the replay program."""
import json
import os
import subprocess

import numpy as np
import pytest
import torch

from helpers import DUBODRA_CONFIGS, ROOT, TraceRun, random_tokens
from plain import dubodra_plain as P

pytestmark = pytest.mark.gpu

TORCH = {"float32": torch.float32, "bfloat16": torch.bfloat16}
NAMES = ["DA", "DB", "DC", "DD"]
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
        _plains[(name, dtype)] = P.PlainDubodra(json.load(open(os.path.join(folder, "config.json"))),
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
    """Rows compared by the root mean square of their difference as a share of the logits' spread: 32-bit within 3e-4
    (the sums' order differs from the float64 model's; the logits of these random models are small numbers, so an absolute
    bound would say little); bfloat16, with the experts' choice agreed (``routed_like_the_engine``), 2.5 % on average and
    not more than one row in fifty beyond 10 %: the token's side input and the joint norm of the linear attention bring
    their input to unit size, so a token whose input happens to be tiny carries its rounding at full size into the stream
    (the plain model with its norms' results rounded to bfloat16 has the same few rows)."""
    err = row_errors(got, ref)
    if dtype == "float32":
        assert float(err.max()) < 3e-4, f"{what}: row errors up to {float(err.max()):.2e} (row {int(err.argmax())})"
        return
    assert float(err.mean()) < 0.025 and float((err > 0.1).double().mean()) <= 0.02, \
        f"{what}: row errors up to {float(err.max()):.3f} (row {int(err.argmax())}), mean {float(err.mean()):.3f}"


class routed_like_the_engine:
    """With random weights a token's best groups or experts are now and then nearly tied, and the bfloat16 engine, whose router
    sees rounded activations, takes another one than the plain model: that row is then off by its whole size, and through
    the recurrent states so are, a little, all rows after it.  So the comparison is done in two halves.  Inside this
    context every choice of the engine's router is recorded (``kernels.moe_route_grouped`` is wrapped); ``logits`` then runs the
    plain model with those choices forced on it (the weights stay its own scores) and checks that the engine's choices are
    the plain model's own wherever the plain model's margin (2 % of a softmax's whole mass) is not small."""

    def __init__(self, monkeypatch):
        from rocmforge_b200 import kernels
        self.calls = []
        real = kernels.moe_route_grouped

        def recording(z, correction, top, **kw):
            idx, w = real(z, correction, top, **kw)
            self.calls.append(idx)
            return idx, w
        monkeypatch.setattr(kernels, "moe_route_grouped", recording)

    def logits(self, plain, tokens, steps=1):
        n_moe = sum((L.get("mlp") or {}).get("kind") == "moe" for L in plain.cfg["layers"])
        assert len(self.calls) == steps * n_moe
        forced = [torch.cat([self.calls[s * n_moe + n] for s in range(steps)]).cpu().long() for n in range(n_moe)]
        seen = []
        out = plain.logits(list(tokens), forced=forced, seen=seen)
        clear = agree = 0
        for mine, (own, margin) in zip(forced, seen):
            sure = margin > 0.02
            clear += int(sure.sum())
            agree += int((mine.sort(dim=-1).values == own.sort(dim=-1).values).all(dim=-1)[sure].sum())
        assert clear == 0 or agree >= 0.995 * clear, f"the engine's router differs from the plain one on {clear - agree} of {clear} clear calls"
        self.calls.clear()
        return out


def vocab(name):
    return DUBODRA_CONFIGS[name]["vocab"]


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
def test_whole_prompt(folders, name, dtype, monkeypatch):
    """Every position of a prompt that crosses four page borders and four chunks of the recurrences."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    toks = random_tokens(vocab(name), 270, 3)
    cache = m.new_cache(max_tokens=512, max_slots=2)
    poison_free_pages(cache)
    s = cache.alloc_slot()
    routes = routed_like_the_engine(monkeypatch)
    got = m.step(cache, [StepRequest(s, toks, range(len(toks)))]).cpu()
    ref = plain_logits(folders, name, dtype, toks) if dtype == "float32" else routes.logits(plain_model(folders, name, dtype), toks)
    close(got, ref, dtype, f"{name} {dtype} whole prompt")


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
            got.append(stream.h.detach().cpu().clone())
        monkeypatch.setattr(block, "forward", recording)
    m.step(cache, [StepRequest(s, toks, range(len(toks)))])
    assert len(got) == len(want)
    for i, (g, w) in enumerate(zip(got, want)):
        assert float((g.double() - w).abs().max()) < 2e-5 * max(1.0, float(w.abs().max())), f"{name}: the stream differs after layer {i}"


@pytest.mark.parametrize("name", ["DA", "DB"])
def test_token_by_token_from_the_first_token(folders, name):
    """One token a step from an empty cache and zero states: the first tokens (fewer than the convolution's taps), page
    borders; and the same logits as the prompt in one step."""
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
def test_portions_of_many_sizes(folders, name, dtype, monkeypatch):
    """A prompt cut into portions of 1 to 70 tokens: the states and the convolution's last inputs are carried from step to
    step (portions shorter than the taps among them), positions count from the sequence's start."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    sizes = [2, 3, 64, 1, 5, 17, 2, 70, 33, 2, 1, 8, 40]
    toks = random_tokens(vocab(name), sum(sizes), 7)
    cache = m.new_cache(max_tokens=512, max_slots=2)
    poison_free_pages(cache)
    s = cache.alloc_slot()
    routes = routed_like_the_engine(monkeypatch)
    got, at = [], 0
    for n in sizes:
        got.append(m.step(cache, [StepRequest(s, toks[at:at + n], range(n))]).cpu())
        at += n
    ref = (plain_logits(folders, name, dtype, toks) if dtype == "float32"
           else routes.logits(plain_model(folders, name, dtype), toks, steps=len(sizes)))
    close(torch.cat(got), ref, dtype, f"{name} {dtype} portions")


def alone(m, tokens, n_prompt):
    """A request through the engine by itself: its prompt in one step, the rest token by token; logits of every position
    from the prompt's last on, and of the prompt's first."""
    from rocmforge_b200 import StepRequest
    cache = m.new_cache(max_tokens=512, max_slots=1)
    s = cache.alloc_slot()
    rows = {}
    first = m.step(cache, [StepRequest(s, tokens[:n_prompt], [0, n_prompt - 1])]).cpu()
    rows[0], rows[n_prompt - 1] = first[0], first[-1]
    for i in range(n_prompt, len(tokens)):
        rows[i] = m.step(cache, [StepRequest(s, [tokens[i]], [0])]).cpu()[0]
    return rows


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", NAMES)
def test_ragged_batch_then_decoding_with_slots_used_again(folders, name, dtype):
    """Unequal prompts in one step (one of a single token, one shorter than the convolution's taps), decoded together;
    requests end at different steps, their slots (two kinds of state and a convolution's inputs) and pages go to new requests; every request must
    equal itself alone: the plain model's logits on the 32-bit path; on the bfloat16 path the engine's own for the
    request by itself (nearly tied experts make single rows of the bfloat16 engine differ from the plain model, see
    ``routed_like_the_engine``; between two schedules of the same engine that is rare, so nine rows in ten must agree to
    2 % and the rest may differ)."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    V = vocab(name)
    lens = [(1, 30), (70, 12), (131, 25), (2, 6)]
    seqs = [random_tokens(V, a + b, 20 + i) for i, (a, b) in enumerate(lens)]
    if dtype == "float32":
        refs = [plain_logits(folders, name, dtype, t) for t in seqs]
    else:
        refs = [alone(m, t, a) for t, (a, _) in zip(seqs, lens)]
    errs = []

    def compare(got, want, what):
        if dtype == "float32":
            close(got, want, dtype, what)
        else:
            errs.extend(row_errors(got, want).tolist())
    cache = m.new_cache(max_tokens=64 * 8, max_slots=4)
    poison_free_pages(cache)
    slots = [cache.alloc_slot() for _ in lens]
    got = m.step(cache, [StepRequest(sl, t[:a], [0, a - 1]) for sl, t, (a, _) in zip(slots, seqs, lens)]).cpu()
    want = torch.stack([r[i] for r, (a, _) in zip(refs, lens) for i in (0, a - 1)])
    compare(got, want, f"{name} {dtype} ragged prompts")
    live = list(range(len(lens)))
    for step in range(30):
        for i in [i for i in live if lens[i][1] <= step]:
            cache.free_slot(slots[i]); live.remove(i)
        poison_free_pages(cache)
        got = m.step(cache, [StepRequest(slots[i], [seqs[i][lens[i][0] + step]], [0]) for i in live]).cpu()
        compare(got, torch.stack([refs[i][lens[i][0] + step] for i in live]), f"{name} {dtype} batch decode step {step}")
    for i in live:
        cache.free_slot(slots[i])
    # the freed slots again: a state or a convolution's inputs that were not zeroed, or a page that
    # kept old keys, would show here
    again = [random_tokens(V, n, 40 + n) for n in (45, 9)]
    slots = [cache.alloc_slot() for _ in again]
    got = m.step(cache, [StepRequest(sl, t, [0, len(t) - 1]) for sl, t in zip(slots, again)]).cpu()
    if dtype == "float32":
        want = torch.cat([plain_logits(folders, name, dtype, t)[[0, len(t) - 1]] for t in again])
    else:
        want = torch.stack([r[i] for t in again for r in [alone(m, t, len(t))] for i in (0, len(t) - 1)])
    compare(got, want, f"{name} {dtype} reused slots")
    if errs:
        errs = torch.tensor(errs)
        assert float((errs < 0.02).double().mean()) >= 0.9 and float(errs.median()) < 0.01, \
            f"{name} bfloat16: batch against alone, median row error {float(errs.median()):.4f}, {int((errs >= 0.02).sum())} of {errs.numel()} rows over 2 %"


def test_a_batch_changes_nothing_beyond_rounding(folders):
    """A request's logits in a batch of unequal requests equal its logits alone up to the order of 32-bit sums (products of
    few tokens cut K into partial sums, products of many do not), in the prompt step and in decoding."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, "DB", "float32")
    V = vocab("DB")
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


@pytest.mark.parametrize("name,dtype", [("DB", "float32"), ("DC", "float32"), ("DC", "bfloat16")])
def test_long_decoding(folders, name, dtype):
    """Three hundred single-token steps after a short prompt, two sequences side by side: the states run on, the attention sees
    every key from the first on.  On the bfloat16 path this is the clustered decode kernel."""
    from rocmforge_b200 import StepRequest
    m = engine(folders, name, dtype)
    a, b = random_tokens(vocab(name), 330, 9), random_tokens(vocab(name), 330, 10)
    cache = m.new_cache(max_tokens=64 * 12, max_slots=2)
    sa, sb = cache.alloc_slot(), cache.alloc_slot()
    got = [m.step(cache, [StepRequest(sa, a[:30], [29]), StepRequest(sb, b[:30], [29])]).cpu()]
    for x, y in zip(a[30:], b[30:]):
        poison_free_pages(cache)
        got.append(m.step(cache, [StepRequest(sa, [x], [0]), StepRequest(sb, [y], [0])]).cpu())
    got = torch.stack(got)
    if dtype == "float32":
        close(got[:, 0], plain_logits(folders, name, dtype, a)[29:], dtype, f"{name} long decoding, first sequence")
        close(got[:, 1], plain_logits(folders, name, dtype, b)[29:], dtype, f"{name} long decoding, second sequence")
        return
    # bfloat16: against the same engine on the whole sequence in one step (the tcgen05 prompt kernel)
    for seq, col in ((a, 0), (b, 1)):
        c2 = m.new_cache(max_tokens=512, max_slots=1)
        whole = m.step(c2, [StepRequest(c2.alloc_slot(), seq, range(29, len(seq)))]).cpu()
        errs = row_errors(got[:, col], whole)
        assert float((errs < 0.03).double().mean()) >= 0.9 and float(errs.median()) < 0.015, \
            f"{name} bfloat16 long decoding: median row error {float(errs.median()):.4f}, worst {float(errs.max()):.3f}"


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_greedy_generation_through_the_public_entry_point(folders, dtype):
    """LLM.generate: the scheduler admits unequal prompts, decode steps replay from graphs (the warm-up run before a
    capture must leave the states as they were), requests end at different lengths."""
    import rocmforge_b200 as rf
    name = "DC"
    llm = rf.LLM(folders(name, dtype), dtype=dtype)
    prompts = [random_tokens(vocab(name), n, 60 + n) for n in (3, 140, 11)]
    out = llm.generate(prompts, max_tokens=12, temperature=0.0, stop_token_ids=[])
    for p, r in zip(prompts, out):
        assert len(r.tokens) == 12
        if dtype == "float32":
            seq = list(p)
            for k, tok in enumerate(r.tokens):
                row = plain_logits(folders, name, dtype, seq)[-1]
                best = int(torch.argmax(row))
                assert tok == best or float(row[best] - row[tok]) <= 1e-5 * float(row.abs().max()), \
                    f"request of {len(p)} tokens, generated token {k}: {tok}, plain {best}"
                seq.append(tok)
        else:
            # bfloat16: against the engine's own step function, token by token without graphs (the plain model may take
            # another expert on a nearly tied token): the generated token is the best one there, or next to it
            from rocmforge_b200 import StepRequest
            cache = llm.model.new_cache(max_tokens=512, max_slots=1)
            s = cache.alloc_slot()
            row = llm.model.step(cache, [StepRequest(s, list(p), [len(p) - 1])]).cpu()[0]
            for tok in r.tokens:
                assert float(row.max() - row[tok]) <= 2e-2 * float(row.abs().max())
                row = llm.model.step(cache, [StepRequest(s, [tok], [0])]).cpu()[0]


def test_command_line(folders):
    """bin/rocmforge on a Dubodra folder: greedy tokens equal the plain model's."""
    folder = folders("DA", "float32")
    prompt = random_tokens(vocab("DA"), 9, 91)
    out = subprocess.run([os.path.join(ROOT, "bin", "rocmforge"), "--model", folder, "--dtype", "float32", "--prompt-ids",
                          ",".join(map(str, prompt)), "--max-tokens", "5", "--temperature", "0", "--stop-ids", "", "--debug"],
                         capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr[-2000:]
    ids = [int(l.split("token_id=")[1]) for l in out.stderr.splitlines() if l.startswith("[Generated]")]
    seq = list(prompt)
    for tok in ids:
        row = plain_logits(folders, "DA", "float32", seq)[-1]
        assert tok == int(torch.argmax(row)) or float(row.max() - row[tok]) <= 1e-5 * float(row.abs().max())
        seq.append(tok)
    assert len(ids) == 5


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_replay_program(folders, tmp_path, dtype):
    """bin/trace_run on a Dubodra folder: whole prompts, a prompt and its last tokens one by one, and a batch."""
    name = "DB"
    V = vocab(name)
    a, b, c = random_tokens(V, 180, 71), random_tokens(V, 37, 72), random_tokens(V, 5, 73)
    ra, rb, rc = (plain_logits(folders, name, dtype, t) for t in (a, b, c))
    tr = TraceRun(folders(name, dtype), dtype, str(tmp_path / "out"), max_tokens=512)

    def ok(got, want, what):
        if dtype == "float32":
            close(got, want, dtype, what)
        else:                                    # rows of a nearly tied expert apart (one expert a token in this model)
            assert float(row_errors(got, want).median()) < 0.03, what
    got = tr.step([("a", a, [0, 6, 7, 99, 100, 179])], end=["a"])
    ok(got, ra[[0, 6, 7, 99, 100, 179]], "replay: whole")
    got = tr.step([("b", b[:30], [29])])
    ok(got, rb[[29]], "replay: prompt")
    for i in range(30, 37):
        got = tr.step([("b", [b[i]], [0])], end=["b"] if i == 36 else [])
        ok(got, rb[[i]], f"replay: decoded {i}")
    got = tr.step([("x", a[:160], [159]), ("y", c[:3], []), ("z", b[:20], [0, 19])])
    ok(got, torch.stack([ra[159], rb[0], rb[19]]), "replay: batch")
    got = tr.step([("x", [a[160]], [0]), ("y", [c[3]], [0]), ("z", [b[20]], [0])], end=["y"])
    ok(got, torch.stack([ra[160], rc[3], rb[20]]), "replay: batch decoded")
    assert tr.step([("x", [a[161]], []), ("z", [b[21]], [])], end=["x", "z"]) is None
    assert tr.close() == 0


