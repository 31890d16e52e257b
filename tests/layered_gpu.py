"""Helpers of the GPU tests of the layer-list decoders: engines, poisoned memory, feeding sequences in portions, tolerances."""
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


def check(got, want, kv, what=""):
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    err = d.pow(2).mean(-1).sqrt() / scale
    worst, typical = float(err.max()), float(err.median())
    assert torch.isfinite(got).all() and worst < TOL[kv][1] and typical < TOL[kv][0], f"{what}: row {int(err.argmax())} of {len(err)} differs by {worst:.3g} (median {typical:.3g})"


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
