"""What every model family's runner shares."""
from __future__ import annotations


class StepOutput:
    __slots__ = ("tokens", "logits", "hidden", "taps", "taps_cat", "read_back")

    def __init__(self, tokens, logits, hidden, taps, taps_cat=None):
        self.tokens, self.logits, self.hidden, self.taps = tokens, logits, hidden, taps
        self.taps_cat = taps_cat        # the tapped hidden states side by side, [rows, taps * H] (taps are views of it)
        self.read_back = None
