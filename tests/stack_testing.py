"""Helpers of the layer-stack tests: tokens, portions, row-wise errors against a plain implementation."""
import torch

TOL = {"fp32": 2e-4, "bf16": 4e-2}


def tokens(cfg, n, seed=5):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def error(got, want):
    """Per row: root mean square of the centred difference over that of the centred reference."""
    d = got.double().cpu() - want
    d, w = d - d.mean(-1, keepdim=True), want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()


def feed(eng, toks, sizes):
    """Logits of every token, fed in portions of the given sizes (the last size repeats)."""
    eng.reset()
    out, at, i = [], 0, 0
    while at < len(toks):
        n = min(sizes[min(i, len(sizes) - 1)], len(toks) - at)
        out.append(eng.extend(toks[at:at + n], list(range(n))))
        at, i = at + n, i + 1
    return torch.cat(out)
