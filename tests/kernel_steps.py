"""Steps for attention kernels called by themselves: requests cut into portions whose keys lie in scattered pages."""
from __future__ import annotations

from types import SimpleNamespace

import numpy as np
import torch


def scrambled_table(totals, page_size, g):
    width = max(-(-t // page_size) for t in totals)
    count = sum(-(-t // page_size) for t in totals) + 3
    order = torch.randperm(count, generator=g).tolist()
    table = torch.full((len(totals), width), -1, dtype=torch.int32)
    for r, t in enumerate(totals):
        for p in range(-(-t // page_size)):
            table[r, p] = order.pop()
    return table, count


def step_of(rows, cache, pieces):
    """The context of a step that brings request r's rows [a, a + n) for (r, a, n) in ``pieces``."""
    index = [(r, a + i) for r, a, n in pieces for i in range(n)]
    step_rows = torch.stack([rows[r][p] for r, p in index]).cuda().contiguous()
    positions = torch.tensor([p for _, p in index], dtype=torch.int32).cuda()
    token_seq = torch.tensor([j for j, (_, _, n) in enumerate(pieces) for _ in range(n)], dtype=torch.int32).cuda()
    starts = torch.tensor(np.concatenate([[0], np.cumsum([n for _, _, n in pieces])]), dtype=torch.int32).cuda()
    sub = type(cache)(cache.need, True, cache.pages, cache.block_table[[r for r, _, _ in pieces]].contiguous(), cache.page_size, None, cache.plane_pages)
    batch = SimpleNamespace(max_q_len=max(n for _, _, n in pieces), num_seqs=len(pieces), max_seq_len=max(a + n for _, a, n in pieces), seq_starts=starts,
                            first_positions=torch.tensor([a for _, a, _ in pieces], dtype=torch.int32).cuda(), num_tokens=len(index), plan=lambda name: None)
    return step_rows, positions, token_seq, sub, batch, index


def pieces_of(lens, firsts):
    """Every request in three steps: rows before ``firsts``, a portion behind them, and its last rows as a step of few rows of their own."""
    tails = [min(n, 3 + r) for r, n in enumerate(lens)]
    return ([(r, 0, f) for r, f in enumerate(firsts) if f > 0], [(r, f, n - t) for r, (n, f, t) in enumerate(zip(lens, firsts, tails)) if n > t],
            [(r, f + n - t, t) for r, (n, f, t) in enumerate(zip(lens, firsts, tails))])
