"""Driving a Session with numpy tokens."""
import numpy as np
import torch


def run(session, portions):
    """portions: token array per row (may be empty).  Logits of all of them, per row."""
    flat = np.concatenate([np.asarray(p, dtype=np.int64) for p in portions])
    hidden = session.extend(torch.from_numpy(flat).cuda(), [len(p) for p in portions])
    logits = session.logits(hidden[: len(flat)]).double().cpu().numpy()
    session.check()
    out, at = [], 0
    for p in portions:
        out.append(logits[at : at + len(p)])
        at += len(p)
    return out


def feed(session, row, ids, sizes):
    """One row's tokens in portions; the logits of all of them."""
    out, at = [], 0
    for n in sizes:
        portions = [[] for _ in range(session.batch)]
        portions[row] = ids[at : at + n]
        out.append(run(session, portions)[row])
        at += n
    assert at == len(ids)
    return np.concatenate(out)


def padded(prompts):
    n = max(len(p) for p in prompts)
    return torch.from_numpy(np.stack([np.concatenate([np.zeros(n - len(p), np.int64), p]) for p in prompts])).cuda()
