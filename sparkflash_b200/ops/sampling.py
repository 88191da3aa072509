"""Candidate filter (top-k / top-p) shared by the engines."""
from __future__ import annotations

import torch

CANDIDATES = 256


def candidate_choice(lg: torch.Tensor, lo: int, world: int, top_k: int, top_p: float, temperature: float, seed: int, pos: int) -> int:
    """One row's next token out of its candidates: every rank offers its CANDIDATES best logits (``lg``: this rank's slice, which
    starts at token ``lo``, banned tokens at -inf) and its slice's log-sum-exp; the union is cut by top-k, then by the nucleus
    over the full-vocabulary softmax, and sampled with a generator keyed on (seed, position), so the choice does not depend on
    batching or speculation.  Reference: candidate gather of the sampler,
    crates/sparkflash-deepseek-forward/src/tp4_forward/sample.rs."""
    T = max(temperature, 1e-5)
    val, idx = torch.topk(lg, min(CANDIDATES, lg.numel()))
    lse = torch.logsumexp(lg / T, 0, keepdim=True)
    idx = idx + lo
    if world > 1:
        import torch.distributed as dist
        vs = [torch.empty_like(val) for _ in range(world)]
        ids = [torch.empty_like(idx) for _ in range(world)]
        ls = [torch.empty_like(lse) for _ in range(world)]
        dist.all_gather(vs, val); dist.all_gather(ids, idx); dist.all_gather(ls, lse)
        val, idx, lse = torch.cat(vs), torch.cat(ids), torch.logsumexp(torch.cat(ls), 0, keepdim=True)
    order = torch.argsort(val, descending=True, stable=True)
    val, idx = val[order], idx[order]
    if temperature < 1e-5:
        return int(idx[0])
    keep = val.numel() if top_k <= 0 else min(top_k, val.numel())
    prob = torch.exp(val / T - lse)                      # probabilities under the full-vocabulary softmax
    if top_p < 1.0:
        before = torch.cumsum(prob, 0) - prob            # mass of the strictly better candidates
        keep = min(keep, max(1, int((before < top_p).sum())))
    prob = prob[:keep]
    g = torch.Generator(device=prob.device)
    g.manual_seed((seed * 0x9E3779B97F4A7C15 + (pos + 1) * 0xBF58476D1CE4E5B9) & 0x7FFFFFFFFFFFFFFF)
    return int(idx[int(torch.multinomial(prob / prob.sum(), 1, generator=g))])
