"""A scheduled step: all-prefill or all-decode (minivllm/scheduler/batch.py:4-12); with
``Config.enable_mixed_steps`` also MIXED: ``requests`` = the prompts to prefill followed by the last
``num_decode`` requests, which decode.

``partial[i]`` marks a prompt of which the step computes a portion only (``Config.enable_chunked_prefill``): it yields
no token.  ``prefill_tokens`` is then the number of prompt tokens of the step."""
import time


class Batch:
    PREFILL, DECODE, MIXED = 0, 1, 2

    def __init__(self, typ: int, reqs: list, num_decode: int = 0):
        self.type = typ
        self.requests = reqs
        self.num_decode = num_decode if typ == Batch.MIXED else (len(reqs) if typ == Batch.DECODE else 0)
        self.mark_partial()
        self.prefill_tokens = None
        self.create_time = time.perf_counter()

    def mark_partial(self) -> None:
        self.partial = [r.portion_end is not None and r.portion_end < len(r.tokens) for r in self.requests]
