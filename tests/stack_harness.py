"""What the tests of the declared stacks share: the runtimes they run on, models and engines over small random checkpoints, feeding a
sequence in portions, paged inputs for single ops, and the comparison with the plain restatement (stack_oracle.py)."""
import json

import numpy as np
import pytest
import torch

import onnxruntime_genai_b200 as og
from stack_models import weights, write
from stack_oracle import stack_forward

RUNTIMES = [pytest.param(("cpu", "float32"), id="cpu"), pytest.param(("cuda", "float32"), id="cuda_fp32", marks=pytest.mark.gpu),
            pytest.param(("cuda", "bfloat16"), id="cuda_bf16", marks=pytest.mark.gpu)]
BLOCK = 16


@pytest.fixture(autouse=True, scope="module")
def one_thread():
    """The matrices here are tiny: more threads than one only wait for each other.  (A test file takes this fixture by importing it.)"""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def tol_of(runtime):
    return 4e-2 if runtime[1] == "bfloat16" else 2e-4


def dtype_of(runtime):
    return torch.bfloat16 if runtime[1] == "bfloat16" else torch.float32


def close(got, want, tol):
    """Root mean square error of every row against the rows' own spread."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape
    err = (got - want).pow(2).mean(-1).sqrt() / want.std()
    assert torch.isfinite(err).all() and float(err.max()) < tol, f"row {int(err.argmax())}: {float(err.max()):.3g} (limit {tol})"


_CACHE = {}


def open_model(tmp_path_factory, name, runtime, cfg, w=None):
    """(model, configuration, weights) of a random checkpoint, opened once per runtime."""
    key = (name, runtime)
    if key not in _CACHE:
        # (16-bit rounding must not decide which experts run: their routers get clear cases)
        w = w or weights(cfg, seed=sum(map(ord, name)), clear_routes=runtime[1] == "bfloat16")
        d = write(cfg, w, tmp_path_factory.mktemp(name))
        c = og.Config(d, provider="cpu" if runtime[0] == "cpu" else "cuda")
        if runtime[0] == "cuda":
            c.set_provider_option("cuda", "compute_dtype", runtime[1])
        _CACHE[key] = (og.Model(c), cfg, w)
    return _CACHE[key]


def open_engine(model, blocks=64, batch=4, tokens=512):
    model.config.overlay(json.dumps({"engine": {"dynamic_batching": {"block_size": BLOCK, "num_blocks": blocks, "max_batch_size": batch,
                                                                     "max_scheduled_tokens": tokens}}}))
    return og.Engine(model)


def random_tokens(cfg, n, seed=0):
    return np.random.RandomState(seed).randint(0, cfg["vocab"], n)


def feed(engine, model, toks, cuts):
    """Logits of every token of one sequence fed in portions of the given sizes (the last size repeats)."""
    r, at, out, i = og.Request(og.GeneratorParams(model)), 0, [], 0
    while at < len(toks):
        n = min(cuts[min(i, len(cuts) - 1)], len(toks) - at)
        out.append(engine.run_given([(r, toks[at:at + n], list(range(n)))])[0])
        at, i = at + n, i + 1
    engine.remove_request(r)
    return torch.cat(out).float().cpu()


def paged(lens, blocks, seed=0):
    """Block tables with shuffled blocks for requests of the given (past, new) lengths; slots and positions of the new tokens."""
    order = np.random.RandomState(seed).permutation(blocks)
    cols = max((p + n + BLOCK - 1) // BLOCK for p, n in lens)
    table, at = np.full((len(lens), cols), -1, dtype=np.int32), 0
    pos, slots = [], []
    for b, (p, n) in enumerate(lens):
        k = (p + n + BLOCK - 1) // BLOCK
        table[b, :k] = order[at:at + k]
        at += k
        pos += list(range(p, p + n))
    cu = np.cumsum([0] + [n for _, n in lens])
    for b, (p, n) in enumerate(lens):
        slots += [int(table[b, q // BLOCK]) * BLOCK + q % BLOCK for q in range(p, p + n)]
    t = lambda x: torch.tensor(np.asarray(x), dtype=torch.int32)
    return dict(table=t(table), pos=t(pos), slots=t(slots), cu=t(cu), past=t([p for p, _ in lens]))


def rows_of(pg, b, n):
    q = np.arange(n)
    return torch.tensor(pg["table"][b].numpy()[q // BLOCK] * BLOCK + q % BLOCK).long()


def wide_rows(x, dev):
    """x [T, n] on the device with rows of whole 16-byte pieces (the form in which projections reach the attention kernels)."""
    out = torch.zeros(x.shape[0], (x.shape[1] + 7) // 8 * 8, dtype=x.dtype, device=dev)[:, :x.shape[1]]
    return out.copy_(x)


def greedy_ok(cfg, w, prompt, generated, tol):
    """Every generated token is the oracle's argmax, or within rounding of it."""
    lg = stack_forward(cfg, w, np.concatenate([prompt, generated]))[0]
    for i, t in enumerate(generated):
        row = lg[len(prompt) - 1 + i]
        assert float(row.max() - row[int(t)]) <= tol * float(lg.std()), f"token {i}"


def beam_search(cfg, w, prompt, n, beams):
    """Plain beam search over the restatement: the best hypothesis of n tokens."""
    hyps = [(0.0, list(map(int, prompt)))]
    while len(hyps[0][1]) < n:
        cand = []
        for score, s in hyps:
            row = torch.log_softmax(stack_forward(cfg, w, s)[0][-1], -1)
            cand += [(score + float(v), s + [int(t)]) for v, t in zip(*torch.topk(row, beams))]
        hyps = sorted(cand, key=lambda c: -c[0])[:beams]
    return np.asarray(hyps[0][1])


def mixed_batches(m, cfg, w, runtime):
    """More requests than fit at once come and go through a pool that is just large enough, portions beside single tokens, requests left
    out of some steps; every request gets the logits it gets alone."""
    eng = open_engine(m, blocks=26, batch=4, tokens=300)
    rng = np.random.RandomState(5)
    waiting = [(i, random_tokens(cfg, n, 20 + i)) for i, n in enumerate((90, 33, 120, 5, 64, 1, 77, 100, 16, 50))]
    live, got, seen, used = [], {i: [] for i, _ in waiting}, dict(waiting), []
    while waiting or live:
        while waiting and len(live) < 4 and sum((len(t) + BLOCK - 1) // BLOCK for _, t, _, _ in live) + (len(waiting[0][1]) + BLOCK - 1) // BLOCK <= 26:
            i, t = waiting.pop(0)
            live.append([i, t, 0, og.Request(og.GeneratorParams(m))])
        step = []
        for e in live:
            if len(live) > 1 and rng.rand() < 0.25:
                continue                                    # left out of this step
            step.append((e, min(int(rng.choice([1, 1, 2, 3, 17, 40, 70])), len(e[1]) - e[2])))
        if not step:
            continue
        out = eng.run_given([(e[3], e[1][e[2]:e[2] + n], list(range(n)) if e[0] % 2 else [n - 1]) for e, n in step])
        eng.core.check_invariants()
        for (e, n), lg in zip(step, out):
            got[e[0]].append((e[2], n, lg.float().cpu()))
            e[2] += n
        for e in [e for e in live if e[2] == len(e[1])]:
            used += e[3]._native.blocks()
            eng.remove_request(e[3])
            live.remove(e)
    assert eng.core.free_blocks == 26 and len(used) > len(set(used))      # blocks were used again
    for i, parts in got.items():
        want = stack_forward(cfg, w, seen[i])[0]
        for at, n, lg in parts:
            close(lg, want[at:at + n] if i % 2 else want[at + n - 1:at + n], 1.5 * tol_of(runtime))


def greedy_generation(m, cfg, w, runtime):
    """Through the generator, and through the scheduler: more requests than the batch holds, prompts cut by a small token budget, blocks that run
    short."""
    tol = 0.2 if runtime[1] == "bfloat16" else 1e-3
    prompts = [random_tokens(cfg, n, 40 + n) for n in (70, 5, 33, 1, 18)]
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=100, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompts[0].astype(np.int32).reshape(1, -1))
    while not gen.is_done():
        gen.generate_next_token()
    solo = np.asarray(gen.get_sequence(0))[70:]
    assert len(solo) == 30
    greedy_ok(cfg, w, prompts[0], solo, tol)
    # the scheduler: more requests than the batch holds, prompts cut by a small token budget, blocks that run short
    eng = open_engine(m, blocks=30, batch=3, tokens=40)
    reqs = []
    for t in prompts:
        gp = og.GeneratorParams(m)
        gp.set_search_options(max_length=len(t) + 25, do_sample=False)
        r = og.Request(gp)
        r.add_tokens(t.astype(np.int32))
        eng.add_request(r)
        reqs.append(r)
    while eng.has_pending_requests():
        r = eng.step()
        if r is None:
            continue
        while r.has_unseen_tokens():
            r.get_unseen_token()
        if r.is_turn_complete():
            r.kept = r.tokens()
            eng.remove_request(r)
    for r, t in zip(reqs, prompts):
        assert len(r.kept) == len(t) + 25
        greedy_ok(cfg, w, t, r.kept[len(t):], tol)


def rewind_and_beams(m, cfg, w, runtime):
    tol = 0.2 if runtime[1] == "bfloat16" else 1e-3
    prompt = np.stack([random_tokens(cfg, 12, 3), random_tokens(cfg, 12, 4)]).astype(np.int32)
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=30, batch_size=2, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompt)
    while not gen.is_done():
        gen.generate_next_token()
    for r in range(2):
        greedy_ok(cfg, w, prompt[r], np.asarray(gen.get_sequence(r))[12:], tol)
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=40, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompt[:1])
    for _ in range(10):
        gen.generate_next_token()
    gen.rewind_to(15)
    for _ in range(7):
        gen.generate_next_token()
    greedy_ok(cfg, w, prompt[0], np.asarray(gen.get_sequence(0))[12:], tol)
    p = og.GeneratorParams(m)
    p.set_search_options(max_length=24, num_beams=3, do_sample=False)
    gen = og.Generator(m, p)
    gen.append_tokens(prompt[:1])
    while not gen.is_done():
        gen.generate_next_token()
    seq = np.asarray(gen.get_sequence(0))
    lp = lambda s: float(sum(torch.log_softmax(stack_forward(cfg, w, s)[0], -1)[i, int(s[i + 1])] for i in range(11, len(s) - 1)))
    # beams follow their own pages: a plain beam search over the restatement finds a hypothesis of the same score (16-bit rounding may pick
    # another one where candidates are close)
    assert abs(lp(seq) - lp(beam_search(cfg, w, prompt[0], 24, 3))) < (4.0 if runtime[1] == "bfloat16" else 2e-2)
