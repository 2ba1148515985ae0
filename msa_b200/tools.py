"""Small host-side helpers shared by the stage-1 worker and the engine front end (mirrors of
``src/utils/tools.py``: ``compose_input`` :101-104, ``RequestLimiter`` :59-99, ``cumulative_concat`` :34-55)."""
from __future__ import annotations

import os
import threading

import torch


def compose_input(doc: str, doc_idx: int, tokenizer):
    """How a memory document is written into a block: ``<|im_start|>[i]. text[i]<|im_end|>`` (src/utils/tools.py:101-104).
    Returns ``(text, tokenizer output)``."""
    new_doc = "<|im_start|>" + f"[{doc_idx}]. {doc}[{doc_idx}]<|im_end|>"
    return new_doc, tokenizer(new_doc, add_special_tokens=False)


class NumberTokenizer:
    """Stands in where a checkpoint has no tokenizer files: text is a list of token ids ("12 7 9"), in both directions."""
    pad_token, pad_token_id, eos_token_id = None, None, None

    def __call__(self, text, add_special_tokens: bool = True, **unused):
        one = isinstance(text, str)
        rows = [[int(w) for w in t.replace(",", " ").split()] for t in ([text] if one else text)]
        mask = [[1] * len(r) for r in rows]
        return {"input_ids": rows[0] if one else rows, "attention_mask": mask[0] if one else mask}

    def batch_decode(self, sequences, **unused):
        return [" ".join(str(int(t)) for t in (s if hasattr(s, "__len__") or getattr(s, "ndim", 0) else [s])) for s in sequences]

    def decode(self, tokens, **unused):
        return self.batch_decode([tokens])[0]


def load_tokenizer(model_path: str):
    """The checkpoint's tokenizer, or ``NumberTokenizer`` when the directory holds none."""
    names = ("tokenizer.json", "tokenizer_config.json", "tokenizer.model", "vocab.json")
    if not any(os.path.exists(os.path.join(model_path, n)) for n in names):
        return NumberTokenizer()
    from transformers import AutoTokenizer
    return AutoTokenizer.from_pretrained(model_path)


def cumulative_concat(tensors):
    """Concatenate per-block id lists that each count from 1 into ids that keep counting across blocks."""
    out, base = [], 0
    for t in tensors:
        out.append(t + base)
        base += int(t[-1])
    return torch.cat(out) if out else torch.empty(0, dtype=torch.long)


class RequestLimiter:
    """At most ``max_concurrent`` requests in flight; ``acquire`` blocks, ``release`` wakes one waiter."""

    def __init__(self, max_concurrent: int = 10):
        self.max_concurrent = max_concurrent
        self.current_count = 0
        self.lock = threading.Lock()
        self.condition = threading.Condition(self.lock)

    def acquire(self) -> bool:
        with self.lock:
            while self.current_count >= self.max_concurrent:
                self.condition.wait()
            self.current_count += 1
            return True

    def release(self) -> None:
        with self.lock:
            if self.current_count > 0:
                self.current_count -= 1
                self.condition.notify()
