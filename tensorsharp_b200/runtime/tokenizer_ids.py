"""Tokenizer of models that come without a vocabulary (model folders): text is the token ids themselves, as decimal numbers
separated by spaces.  A word that is not the number of a token is taken by its UTF-8 bytes (modulo the vocabulary size), so
that any prompt can be run.  There is no end-of-sequence token."""
from __future__ import annotations

from typing import Iterable, List


class IdTokenizer:
    def __init__(self, vocab_size: int):
        self.vocab_size = int(vocab_size)
        self.eos_id = -1

    def is_eos(self, tid: int) -> bool:
        return False

    def lookup_token(self, s: str) -> int:
        return int(s) if s.isascii() and s.isdigit() and int(s) < self.vocab_size else -1

    def encode(self, text: str, add_special: bool = True) -> List[int]:
        out: List[int] = []
        for word in text.split():
            t = self.lookup_token(word)
            out += [t] if t >= 0 else [b % self.vocab_size for b in word.encode("utf-8")]
        return out

    def token_bytes(self, tid: int) -> bytes:
        return f"{int(tid)} ".encode()

    def decode(self, ids: Iterable[int]) -> str:
        return " ".join(str(int(t)) for t in ids)
