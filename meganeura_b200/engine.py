"""Step-by-step execution of a row-dynamic model (one sequence at a time): the tokens of a prompt in
portions, single tokens from a captured CUDA graph, greedy generation with the pick on the device.
"""
from __future__ import annotations

import numpy as np

from ._lib import ROWS_PICKED, ROWS_TOKENS


class Engine:
    def __init__(self, model, greedy: bool = True):
        """greedy: pick the next token on the device after every step that computes logits (generate
        needs it; feed works with and without)."""
        self.model, self.session = model, model.session
        self.vocab = model.cfg.vocab
        self.pos = 0
        self.greedy = greedy
        self._single_steps = 0
        self._captured = False
        if greedy:
            self.session.enable_greedy(0, "token_ids", "kv_pos", model.max_tokens)

    def end(self) -> None:
        """Finish the sequence: its recurrent state and cache are given back (cleared)."""
        self.session.reset_state()
        self.pos = 0

    def _check(self, tokens) -> np.ndarray:
        tokens = np.asarray(tokens, dtype=np.int64).reshape(-1)
        if tokens.size and (tokens.min() < 0 or tokens.max() >= self.vocab):
            raise ValueError(f"token ids must lie in [0, {self.vocab})")
        if self.pos + tokens.size > self.model.max_tokens:
            raise ValueError(f"{self.pos + tokens.size} tokens exceed the session's limit of {self.model.max_tokens}")
        return tokens.astype(np.uint32)

    def _step(self, tokens: np.ndarray, picked) -> None:
        """One session step; logits of `picked` rows are left in the session's output."""
        s = self.session
        s.set_rows(ROWS_TOKENS, len(tokens))
        s.set_rows(ROWS_PICKED, len(picked))
        s.set_input_u32("token_ids", tokens)
        s.set_input_u32("kv_pos", [self.pos])
        if len(picked):
            s.set_input_u32("picked_rows", picked)
        s.step()
        self.pos += len(tokens)
        self._after_step(len(tokens), len(picked))

    def _after_step(self, rows: int, picked: int) -> None:
        # a captured step needs its kernels to have run once (their attributes are set at the first launch)
        if rows == 1 and picked == 1 and not self._captured:
            self._single_steps += 1
            if self._single_steps >= 2:
                self.session.capture()
                self._captured = True

    def feed(self, tokens, want=()) -> np.ndarray:
        """Continue the sequence by `tokens`; returns the logits [len(want), vocab] at the places `want`
        among them, in the order of `want`."""
        tokens = self._check(tokens)
        want = np.asarray(want, dtype=np.int64).reshape(-1)
        if want.size and (want.min() < 0 or want.max() >= tokens.size):
            raise ValueError("a wanted place lies outside the tokens")
        out = np.empty((want.size, self.vocab), dtype=np.float32)
        rows, picks = self.model.max_rows, self.model.max_picked
        at = 0
        while at < tokens.size:
            n = min(rows, tokens.size - at)
            while True:                                    # a portion ends where its wanted rows still fit
                mine = np.nonzero((want >= at) & (want < at + n))[0]
                if mine.size <= picks or n == 1:
                    break
                n = max(1, n // 2)
            places = np.unique(want[mine])                 # a place asked for twice is computed once
            self._step(tokens[at:at + n], (places - at).astype(np.uint32))
            if places.size:
                self.session.wait()
                logits = self.session.read_output(places.size * self.vocab).reshape(places.size, self.vocab)
                out[mine] = logits[np.searchsorted(places, want[mine])]
            at += n
        self.session.wait()
        return out

    def generate(self, prompt, max_new: int) -> np.ndarray:
        """Greedy continuation of the sequence by `prompt` and max_new picked tokens (the last one is not
        fed): the pick runs on the device and feeds the next step."""
        prompt = self._check(prompt)
        if prompt.size == 0 or max_new < 1:
            raise ValueError("a prompt and at least one new token are needed")
        if self.pos + prompt.size + max_new - 1 > self.model.max_tokens:
            raise ValueError(f"{self.pos + prompt.size + max_new - 1} tokens exceed the session's limit of {self.model.max_tokens}")
        s, rows = self.session, self.model.max_rows
        if not self.greedy:
            raise RuntimeError("this engine was made without the greedy pick")
        start = self.pos
        for at in range(0, prompt.size, rows):
            part = prompt[at:at + rows]
            last = at + part.size == prompt.size
            self._step(part, np.array([part.size - 1], np.uint32) if last else [])
        s.set_rows(ROWS_TOKENS, 1)
        s.set_rows(ROWS_PICKED, 1)
        s.set_input_u32("picked_rows", [0])
        for _ in range(max_new - 1):
            s.step()
            self.pos += 1
            self._after_step(1, 1)
        return s.read_tokens(start + prompt.size - 1, max_new)
