"""Masks of causal attention. An int is a run length: token i sees the tokens j <= i of its own run of so many positions, counted
from 0 (0: it sees all of them). ``Window``: token i sees the tokens j with 0 <= i - j < size."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Union


@dataclass(frozen=True)
class Window:
    size: int

    def __post_init__(self):
        if self.size < 1:
            raise ValueError("a window holds at least the token itself")


Mask = Union[int, Window]
