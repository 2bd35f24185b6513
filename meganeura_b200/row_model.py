"""What the row-dynamic decoders share: one sequence's session over a graph whose step may hold a whole
prompt, a portion or a single token; weights by name, bf16 on the device; operand precision by dtype.
"""
from __future__ import annotations

import numpy as np

from ._lib import FMT_BF16, FMT_F32, ROWS_PICKED, ROWS_TOKENS
from .graph import Graph, Session, build_inference_session


class RowModel:
    """max_rows: tokens of the largest step; max_picked: most rows of a step whose logits are read;
    max_tokens: positions a sequence may reach.  tap_layers: the residual stream after every layer becomes
    an output too (indices 1.. of read_output_by_index).  A subclass builds its graph in _build(), which
    appends each layer's output to self._taps and returns the logits."""

    def __init__(self, cfg, dtype: str = "bfloat16", max_rows: int = 512, max_picked: int = 256, max_tokens: int = 4096, lora_rank=None,
                 tap_layers: bool = False):
        """lora_rank: {layer or tensor prefix: rows of its low-rank decay projection}."""
        if dtype not in ("bfloat16", "float32"):
            raise ValueError(f"dtype must be bfloat16 or float32, not {dtype}")
        self.cfg, self.dtype = cfg, dtype
        self.max_rows, self.max_picked, self.max_tokens = min(max_rows, max_tokens), min(max_picked, max_rows, max_tokens), max_tokens
        self.lora_rank = lora_rank or {}
        self._params, self._nodes = [], {}                     # (name, shape, bf16?), name -> node
        self._operand = FMT_BF16 if dtype == "bfloat16" else FMT_F32
        self.graph = Graph()
        self._taps = []
        self.token_ids = self.graph.input_u32_rows("token_ids", self.max_rows, ROWS_TOKENS)
        self.picked = self.graph.input_u32_rows("picked_rows", self.max_picked, ROWS_PICKED)
        self.pos = self.graph.input_u32("kv_pos", [1])
        logits = self._build(self.graph)
        self.graph.set_outputs([logits] + (self._taps if tap_layers else []))
        self.session: Session = build_inference_session(self.graph)

    def _build(self, g: Graph) -> int:
        raise NotImplementedError

    # ---- weights as graph nodes; a name asked for again (layers that share weights) is the same node
    def _vec(self, name, n):
        if name not in self._nodes:
            self._params.append((name, (n,), False))
            self._nodes[name] = self.graph.parameter(name, [n])
        return self._nodes[name]

    def _mat(self, name, n, k):
        if name not in self._nodes:
            self._params.append((name, (n, k), True))
            self._nodes[name] = self.graph.parameter_bf16(name, [n, k])
        return self._nodes[name]

    def _linear(self, x, name, n, k, bias=None):
        y = self.graph.matmul_bt(x, self._mat(name, n, k))
        return y if bias is None else self.graph.bias_add(y, self._vec(bias, n))

    def parameters(self):
        """(name, shape, stored as bf16 on the device) of every weight."""
        return list(self._params)

    def load(self, tensors) -> None:
        """tensors: a weights.SafeTensors, or anything with shape / dtype / raw / f32 of the names."""
        for name, shape, bf16 in self._params:
            have = tuple(tensors.shape(name))
            if int(np.prod(have)) != int(np.prod(shape)) or (bf16 and have != tuple(shape)):
                raise ValueError(f"tensor '{name}' has the shape {list(have)}, the configuration needs {list(shape)}")
            if bf16 and tensors.dtype(name) == "BF16":
                self.session.upload_param(name, tensors.raw(name))
            else:
                self.session.set_parameter(name, tensors.f32(name))
