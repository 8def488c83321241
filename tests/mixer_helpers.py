"""Helpers for GPU tests of parts on their own: a step context, a cache for a few mixers, random parameters."""
import torch


def make_ctx(entries, slots=None, max_tokens=1024, max_requests=8, widths=()):
    """A step context for [(pos0, n tokens)] entries, with explicit block tables per group."""
    from ferrum_b200.engine.batch import StepContext, StepEntry
    ctx = StepContext("cuda", max_tokens, max_requests, [len(t[0]) for t in widths])
    es = [StepEntry(slots[i] if slots else i, p0, list(range(n))) for i, (p0, n) in enumerate(entries)]
    ctx.fill(es, [list(t) for t in widths])
    return ctx


class SomeMixers:
    """The least a cache needs of a model: a schedule and the needs of its runs."""

    def __init__(self, mixers):
        from ferrum_b200.models import Run
        self.mixers, self.schedule = mixers, [Run(i) for i in range(len(mixers))]

    def cache_needs(self):
        return [m.cache_need() for m in self.mixers]


def fill_part(part, seed, td, prefix, short_name, std=0.3, fixed=None):
    """Random parameters for a part and its children; returns them under the plain implementation's names
    (`short_name` of a part's name; float64)."""
    from ferrum_b200.weights.random_init import _tensor
    w = {}
    for name, ps, owner, local in part.named_specs():
        t = _tensor(f"{prefix}{name}", ps, seed, "cuda", std if ps.kind == "matrix" else 0.2)
        if fixed and name in fixed:
            t = fixed[name].to("cuda")
        t = t.to(td) if ps.kind == "matrix" else t.float()
        owner.assign(local, t.contiguous())
        w[prefix + short_name(name)] = t.double().cpu()
    part.finalize()
    return w


def run_mixers_in_portions(mixers, xs, cuts, td, max_tokens=128, page=8):
    """The mixers one after another on rows of their own in every step (as the layers of a model run)."""
    from ferrum_b200.cache import CacheStorage
    from ferrum_b200.engine.batch import StepContext, StepEntry
    cache = CacheStorage(SomeMixers(mixers), td, "cuda", page_size=page, max_tokens=max_tokens, max_requests=3, max_model_len=max_tokens)
    ctx = StepContext("cuda", max_tokens, 3, [cache.table_width] * cache.n_groups)
    cache.open()                              # the request under test takes the second slot
    slot = cache.open()
    for s in cache.states:
        s[slot].fill_(float("nan"))           # a state row that a first token must not read
    got, at = [[] for _ in mixers], 0
    for n in cuts:
        cache.manager.grow(slot, at + n)
        if at == 0:
            for s in cache.states:
                s[slot].zero_()               # (what the step function does for a request's first tokens)
        ctx.fill([StepEntry(slot, at, list(range(n)))], cache.manager if cache.n_groups else [])
        for i, (mx, x) in enumerate(zip(mixers, xs)):
            y = torch.zeros(n, x.shape[1], device="cuda")
            mx.forward(x[at:at + n].contiguous(), ctx, cache.layer_cache(i), y, accumulate=False)
            got[i].append(y.double().cpu())
        assert ctx.err.item() == 0
        cache.manager.commit(slot, at + n)
        at += n
    return [torch.cat(g) for g in got]
