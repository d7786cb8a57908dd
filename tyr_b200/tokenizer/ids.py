"""Token ids written as text, for checkpoints without a tokenizer: ``"5 17 3"`` <-> ``[5, 17, 3]``."""
from __future__ import annotations

from typing import List, Optional, Sequence


class IdTokenizer:
    def __init__(self, vocab: int):
        self.vocab = vocab

    def encode(self, text: str) -> List[int]:
        try:
            ids = [int(t) for t in text.replace(",", " ").split()]
        except ValueError:
            raise ValueError(f"this checkpoint has no tokenizer: a prompt is a list of token ids, got {text!r}") from None
        bad = [i for i in ids if not 0 <= i < self.vocab]
        if bad or not ids:
            raise ValueError(f"token ids must be between 0 and {self.vocab - 1}, got {bad}" if bad else "empty prompt")
        return ids

    def decode(self, ids: Sequence[int], skip_special: bool = True) -> str:
        return "".join(f"{int(i)} " for i in ids)

    def token_id(self, token: str) -> Optional[int]:
        return None
