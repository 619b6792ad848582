"""Shared by the tests of step engines: sequences in portions, batches of sequences, distances between logits."""
import torch


def run_cuts(eng, slot, ids, cuts):
    """One sequence in portions; returns the logits of every position."""
    from neuralfn_b200.serving import StepEntry
    eng.release(slot)
    out, at = [], 0
    for n in cuts:
        part = ids[at:at + n]
        out.append(eng.step([StepEntry(slot, part, range(len(part)))], logits=True)[1])
        at += n
    assert at == len(ids)
    return torch.cat(out)


def worst(got, want):
    d = got.double() - want
    d = d - d.mean(-1, keepdim=True)
    spread = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return float((d.pow(2).mean(-1).sqrt() / spread).max())


def repeat_cuts(n, sizes):
    out, left, i = [], n, 0
    while left:
        k = min(sizes[i % len(sizes)], left)
        out.append(k)
        left -= k
        i += 1
    return out


def run_mixed(eng, seqs, *, slots, room, seed, sizes=(1, 1, 2, 19, 50)):
    """Unequal requests together, some fed by portions and some by single tokens, left out of steps, ended and replaced in a pool that
    holds `room` tokens of live requests; returns every request's logits."""
    from neuralfn_b200.serving import StepEntry
    g = torch.Generator().manual_seed(seed)
    waiting, live, free, at = list(range(len(seqs))), {}, list(range(slots)), {}
    got = [[] for _ in seqs]
    held = lambda i: (len(seqs[i]) + 63) // 64 * 64  # noqa: E731
    while waiting or live:
        for i in list(waiting):
            if free and sum(held(k) for k in live) + held(i) <= room:
                live[i], at[i] = free.pop(), 0
                eng.release(live[i])
                waiting.remove(i)
        entries, who = [], []
        for i, slot in live.items():
            kind = int(torch.randint(0, len(sizes), (1,), generator=g))
            if kind == 0 and len(live) > 1 and entries:
                continue
            n = min(sizes[kind], len(seqs[i]) - at[i])
            entries.append(StepEntry(slot, seqs[i][at[i]:at[i] + n], range(n)))
            who.append((i, n))
        rows = eng.step(entries, logits=True)[1]
        base = 0
        for i, n in who:
            got[i].append(rows[base:base + n])
            base += n
            at[i] += n
            if at[i] == len(seqs[i]):
                eng.release(live[i])
                free.append(live.pop(i))
    return [torch.cat(x) for x in got]
