"""Running a batch step by step with token ids that the caller supplies.

``BatchSteps`` is the token loop of ``GenerationMixin`` without its sampling: a padded prompt call that fills a
``StaticKVCache``, then one token per sequence and call. Everything between two choices of a token - the inputs of the
call, padding and mask, cache and state, the rows that go on - is the code ``generate()`` uses.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence

import torch
from torch import Tensor


class BatchSteps:
    """``steps = BatchSteps(model); steps.start([ids_a, ids_b]); steps.advance([tok_a, tok_b]); steps.keep([1])``.

    Prompts of different lengths are padded on the left, as ``generate()`` expects them. ``logits`` of ``start`` / ``advance``
    have one row of positions per sequence; position ``i`` of sequence ``r``'s prompt is column ``pad[r] + i``.
    """

    def __init__(self, model, reserve: int = 256) -> None:
        self.model = model
        self.reserve = int(reserve)
        self.kwargs: Dict[str, Any] = {}
        self.ids: Optional[Tensor] = None
        self.pad: List[int] = []

    @property
    def rows(self) -> int:
        return 0 if self.ids is None else self.ids.size(0)

    def _call(self, last_only: bool) -> Tensor:
        inputs = self.model.prepare_inputs_for_generation(self.ids, **self.kwargs)
        out = self.model(**inputs, return_dict=True, last_token_logits=last_only)
        self.kwargs = self.model._update_model_kwargs_for_generation(out, self.kwargs)
        return out["logits"]

    @torch.no_grad()
    def start(self, prompts: Sequence[Sequence[int]], last_only: bool = False) -> Tensor:
        """The first call of a batch; returns logits ``[rows, longest prompt, vocab]`` (``last_only``: of the last position)."""
        from ..models.common import StaticKVCache
        if self.ids is not None:
            raise RuntimeError("this batch has been started already")
        if not prompts or any(len(p) == 0 for p in prompts):
            raise ValueError("every sequence of a batch needs at least one token")
        dev, longest = self.model.device, max(len(p) for p in prompts)
        self.pad = [longest - len(p) for p in prompts]
        self.ids = torch.tensor([[0] * n + list(p) for n, p in zip(self.pad, prompts)], dtype=torch.long, device=dev)
        mask = torch.tensor([[0] * n + [1] * len(p) for n, p in zip(self.pad, prompts)], dtype=torch.long, device=dev)
        self.kwargs = {"past_key_values": StaticKVCache(longest + self.reserve, grow=True), "attention_mask": mask, "use_cache": True}
        return self._call(last_only)

    @torch.no_grad()
    def advance(self, tokens: Sequence[int]) -> Tensor:
        """One more token per sequence; returns logits ``[rows, 1, vocab]``."""
        if self.ids is None or len(tokens) != self.rows:
            raise ValueError(f"{self.rows} sequences, {len(tokens)} tokens")
        new = torch.tensor(list(tokens), dtype=torch.long, device=self.ids.device)
        self.ids = torch.cat([self.ids, new[:, None]], dim=-1)
        return self._call(True)

    def keep(self, rows: Sequence[int]) -> None:
        """Go on with these sequences only; what the others held in the cache is given back."""
        if list(rows) == list(range(self.rows)):
            return
        at = torch.tensor(list(rows), dtype=torch.long, device=self.ids.device)
        self.pad = [self.pad[r] for r in rows]
        self.ids = self.ids.index_select(0, at)
        self.kwargs["past_key_values"] = self.model._reorder_cache(self.kwargs["past_key_values"], at)
        for name in ("attention_mask", "token_type_ids", "position_ids"):
            if self.kwargs.get(name) is not None:
                self.kwargs[name] = self.kwargs[name].index_select(0, at)
