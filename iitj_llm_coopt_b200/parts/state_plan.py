"""The per-step plan of the mixers with a matrix state per head (`Kernels.matrix_memory`, `Kernels.gated_delta`): which requests of the
step are walked token by token and which bring a portion long enough to be cut into chunks of neighbouring tokens that are worked on as
matrix products.  Every such layer of a model shares one plan per step."""
from __future__ import annotations

from .base import StepPlan

KEY = "matrix_state"


def plan_state_chunks(kernels, shape):
    """StepPlan with `walks` (requests), `chunks` (request, first token row, tokens, index of the chunk in its request) and `longs`
    (request, first chunk, chunks), and their counts on the host; None for a step of single tokens or a kernel set without chunks."""
    size = getattr(kernels, "STATE_CHUNK", 0)
    if not size or shape.num_tokens == len(shape.query_lens):
        return None
    walks, chunks, longs, row = [], [], [], 0
    for b, n in enumerate(shape.query_lens):
        if n >= kernels.state_chunk_from:
            longs += [b, len(chunks) // 4, -(-n // size)]
            for j, s in enumerate(range(0, n, size)):
                chunks += [b, row + s, min(size, n - s), j]
        elif n:
            walks.append(b)
        row += n
    counts = (len(walks), len(chunks) // 4, len(longs) // 3)
    plan = StepPlan(arrays={"walks": walks or [0], "chunks": chunks or [0], "longs": longs or [0]}, graph_key=counts)
    plan.counts = counts
    return plan
