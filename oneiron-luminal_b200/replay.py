"""Replays a trace of request portions through the runtime and hands back logits: no sampling, the generation path's own step.

Requests live in the sequences of a paged cache; every step runs only the tokens it brings, at the position its request has reached.
"""
from __future__ import annotations

from typing import Dict, Iterable, List

PAGE_ROWS = 64


class TraceReplay:
    def __init__(self, rt, slots: int):
        self.rt = rt
        self.free: List[int] = list(range(slots))[::-1]
        self.slot: Dict[str, int] = {}
        self.pos: Dict[str, int] = {}

    @staticmethod
    def capacity(max_tokens: int, slots: int = 16) -> dict:
        """``from_config`` keywords for a cache that holds ``max_tokens`` tokens of live requests (each ends in a partial page)."""
        pages = -(-max(1, max_tokens) // PAGE_ROWS)
        return dict(max_seq=pages * PAGE_ROWS, max_batch=slots, kv_page_rows=PAGE_ROWS, kv_pool_pages=pages + slots, max_new_tokens=16)

    def step(self, entries: Iterable[dict], end: Iterable[str]) -> List:
        """Runs each entry's tokens; returns one logits row per wanted place, in the order of the entries and of their ``want``."""
        rt, rows = self.rt, []
        for e in entries:
            rid, tokens, want = e["id"], e["tokens"], e["want"]
            if rid not in self.slot:
                if not self.free:
                    raise RuntimeError("more live requests than cache slots")
                self.slot[rid], self.pos[rid] = self.free.pop(), 0
            if not tokens:
                continue
            rt.seq_select(self.slot[rid])
            places = sorted(set(want))
            rt.want_logits(places)
            rt.set_data(tokens)
            rt.execute({"s": len(tokens), "p": self.pos[rid]})
            self.pos[rid] += len(tokens)
            if places:
                got = rt.get_wanted()
                rows += [got[places.index(w)] for w in want]
        for rid in end:
            if rid in self.slot:
                slot = self.slot.pop(rid)
                rt.kv_release(slot)
                self.free.append(slot)
                del self.pos[rid]
        rt.synchronize()
        return rows
