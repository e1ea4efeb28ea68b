"""How the rows of a step are cut into chunks, for recurrences that work on chunks of long portions."""
from __future__ import annotations

import torch


def chunk_layout(ctx, chunk: int):
    """(chunks of all rows before each row [rows] int32 on the device, chunks of all rows, most chunks of a row), worked out once per
    step and chunk length."""
    def make():
        counts = [-(-n // chunk) for n in ctx.host["q_lens"]]
        base = [sum(counts[:i]) for i in range(len(counts))]
        return torch.tensor(base, dtype=torch.int32).to(ctx.device, non_blocking=True), sum(counts), max(counts)
    return ctx.memo(("chunk layout", chunk), make)
