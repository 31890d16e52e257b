"""Helpers of the GPU tests of the layer-list decoders: engines, poisoned memory, feeding sequences in portions, tolerances."""
import numpy as np
import torch

# rms error of a logits row over the rms of all rows (means taken off): median and worst row.  A recurrence divides by a sum
# that can come near zero; such rows amplify rounding ten- to thirtyfold in either mode.
TOL = {"f32": (4e-6, 2e-4), "bf16": (0.015, 0.15)}


def engine(model, kv, max_batch=4, max_seq=384, pages=None, chunk=512):
    from oxibonsai_b200.runtime import EngineBuilder
    return (EngineBuilder().model_path(model.path).preset("greedy").max_seq_len(max_seq).max_batch(max_batch).kv_cache(kv, 64, pages)
            .prefill_chunk(chunk).build())


def poison(eng):
    """Everything a sequence must not read becomes NaN: free cache rows, key factors and recurrent state."""
    for d in (eng.kv.rows, eng.kv.values, eng.kv.factors):
        for t in d.values():
            t.fill_(float("nan"))
    for d in eng.runner.states.tensors.values():
        for t in d.values():
            t.fill_(float("nan"))


def check(got, want, kv, what="", tol=None):
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    err = d.pow(2).mean(-1).sqrt() / scale
    worst, typical = float(err.max()), float(err.median())
    tol = TOL[kv] if tol is None else tol[kv]
    assert torch.isfinite(got).all() and worst < tol[1] and typical < tol[0], f"{what}: row {int(err.argmax())} of {len(err)} differs by {worst:.3g} (median {typical:.3g})"


def feed(eng, tokens, cuts, slot=0, close=True):
    """Runs one sequence in portions of the given sizes (the rest in one); logits of every position."""
    out, at = [], 0
    for n in list(cuts) + [len(tokens)]:
        n = min(n, len(tokens) - at)
        if n > 0:
            eng.reserve(slot, at + n)
            out.append(eng.feed([(slot, tokens[at:at + n], at)], [list(range(n))]).clone())
            at += n
    if close:
        eng.close_sequence(slot)
    return torch.cat(out)


def run_unequal_requests(model, eng, kv, tol=None):
    """Unequal requests over four slots: portions beside decoded tokens, left out now and then, ending at different times; pages
    and slots are used again, over memory that starts full of NaN.  Every position is compared with the request alone."""
    poison(eng)
    rng = np.random.default_rng(7)
    reqs = [model.tokens(n, seed=20 + n) for n in (3, 130, 1, 77, 201, 64, 40, 65)]
    want = [model.logits(t) for t in reqs]
    queue, live, free, got = list(range(len(reqs))), {}, [2, 0, 3, 1], {i: [] for i in range(len(reqs))}
    while queue or live:
        while queue and free and len(live) < 4:
            live[queue.pop(0)] = [free.pop(0), 0]
        chosen = [i for i in live if rng.random() < 0.8] or list(live)
        entries, wants, lens = [], [], []
        for i in chosen:
            slot, at = live[i]
            n = min(int(rng.choice([1, 1, 2, 3, 17, 60])), len(reqs[i]) - at)
            eng.reserve(slot, at + n)
            entries.append((slot, reqs[i][at:at + n], at))
            wants.append(list(range(n)))
            lens.append(n)
        out = eng.feed(entries, wants).clone()
        for i, part in zip(chosen, out.split(lens)):
            got[i].append(part)
            live[i][1] += len(part)
            if live[i][1] == len(reqs[i]):
                eng.close_sequence(live[i][0])
                free.append(live.pop(i)[0])
    for i in got:
        check(torch.cat(got[i]), want[i], kv, what=f"request {i}", tol=tol)
