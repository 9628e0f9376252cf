"""What the tests of the layer-stack families share."""

import numpy as np


def portions(model, ids, sizes):
    """Logits of every position, fed in portions of the given sizes over and over."""
    out, at, i = [], 0, 0
    while at < len(ids):
        n = min(sizes[i % len(sizes)], len(ids) - at)
        out.append(model.feed(ids[at:at + n], at, range(n)))
        at, i = at + n, i + 1
    return np.concatenate(out)


def pad(a, ld):
    out = np.zeros((a.shape[0], ld), a.dtype)
    out[:, :a.shape[1]] = a
    return out


def bf16_array(bits):
    return (np.asarray(bits, np.uint16).astype(np.uint32) << 16).view(np.float32)


def follows(forward, cfg, w, prompt, ids, tol):
    """Every generated token is the oracle's best for the sequence so far, or within rounding of it."""
    lg, _ = forward(cfg, w, np.concatenate([prompt, ids]))
    for i, t in enumerate(ids):
        row = lg[len(prompt) - 1 + i]
        assert row.max() - row[t] <= tol * np.std(row), i
