"""The serving engine over one configuration of a family of ``models/registry.py``, fed by trace steps: shared by the model tests."""
import torch


def logit_error(got, want):
    """Largest rms difference of a row of logits, mean taken off, over the spread of the wanted logits."""
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / want.std()).max())


def cut(rnd, n, sizes):
    """``n`` in portions of random sizes."""
    out = []
    while n:
        c = min(n, rnd.choice(sizes))
        out.append(c)
        n -= c
    return out


class Rig:
    """``run`` feeds steps of (request, count) and returns each request's logits of every row."""

    def __init__(self, cfg, weights, dtype, *, context=320, pool=0, residents=4, rows=256, graphs=True):
        from ironpangu_b200.models import registry
        from ironpangu_b200.parallel.fabric import Fabric
        from ironpangu_b200.runtime.engine_worker import BatchEngine

        fam = next(f for f in registry.FAMILIES if f.architecture == cfg["architecture"])
        mod = fam.load()
        self.cfg, self.fab, self.w = cfg, Fabric(0, 1), weights
        config = getattr(mod, fam.architecture + "Config").from_dict(cfg)
        self.dec = getattr(mod, fam.decoder)(config, self.w, self.fab, max_context=context, num_slots=residents, pool_tokens=pool, keep_logits=True, dtype=dtype)
        self.eng = BatchEngine(self.dec, "t", context, cfg["vocab"], prefill=getattr(mod, fam.rows)(self.dec, max_rows=rows), use_graphs=graphs)

    def run(self, requests, steps):
        """requests: id -> tokens; steps: lists of (id, count). A request ends with its last token; ids with '#' run the tokens of the
        part before it once more."""
        from ironpangu_b200.runtime.replay import Replay

        r, at, out = Replay(self.eng), {}, {}
        for n, step in enumerate(steps):
            entries, end, got = [], [], []
            for name, count in step:
                toks = requests[name.split("#")[0]]
                lo = at.get(name, 0)
                part = toks[lo:lo + count]
                entries.append({"id": name, "tokens": part, "want": list(range(len(part)))})
                got += [name] * len(part)
                at[name] = lo + len(part)
                if at[name] == len(toks):
                    end.append(name)
            logits = r.step({"step": n, "entries": entries, "end": end})
            for i, name in enumerate(got):
                out.setdefault(name, []).append(logits[i])
        assert self.fab.status() == 0
        return {k: torch.stack(v) for k, v in out.items()}

    def close(self):
        self.dec.state_manager.close()
        self.fab.close()


def random_batches(rnd, lens, order, live_most, pool_tokens, sizes):
    """Steps of up to ``live_most`` requests (``lens``: id -> tokens, '#' ids use the part before it) that hold at most ``pool_tokens``
    rounded up to 64 each; requests are left out of some steps."""
    size = lambda k: lens[k.split("#")[0]]
    waiting, live, steps = list(order), {}, []
    while waiting or live:
        while waiting and len(live) < live_most and sum((size(k) + 63) // 64 * 64 for k in list(live) + waiting[:1]) <= pool_tokens:
            k = waiting.pop(0)
            live[k] = size(k)
        step = []
        for k in list(live):
            if rnd.random() < 0.2:
                continue
            c = min(live[k], rnd.choice(sizes))
            step.append((k, c))
            live[k] -= c
            if not live[k]:
                del live[k]
        if step:
            steps.append(step)
    return steps
