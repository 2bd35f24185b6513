"""Tobovik: a decoder of gated linear attention ('gla') layers and of layers that run softmax attention and
gated linear attention side by side on one input ('parallel'), each followed by an optional SiLU GLU.
Sinusoidal positions are added to the embedding; the sublayers read the residual stream itself and their
outputs are normed before they are added; a layer may use an earlier layer's weights with state and cache
of its own.

Every size and constant comes from config.json or a tensor's shape.  Weights stay bf16 on the device; with
dtype float32 the activations, caches and matrix products are f32, with bfloat16 the operands of the linear
layers are bf16 and the key / value caches f16 (positions, norms, decays, recurrent state, attention scores
and the residual stream are f32 in both).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from ._lib import FMT_BF16, GATE_SIGMOID, GATE_SILU, lib
from .graph import Graph
from .row_model import RowModel

POSITION_BASE = 10000.0      # fixed by the design


@dataclass(frozen=True)
class GlaConfig:
    heads: int
    dim: int                             # query / key dimensions of a head
    vdim: int
    tau: float

    @staticmethod
    def from_dict(m: dict) -> "GlaConfig":
        return GlaConfig(int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["tau"]))


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    temp_coef: float
    temp_every: float

    @staticmethod
    def from_dict(m: dict) -> "AttentionConfig":
        a = AttentionConfig(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), float(m["q_temp"]["coef"]),
                            float(m["q_temp"]["every"]))
        if a.kv_heads < 1 or a.heads % a.kv_heads:
            raise ValueError(f"{a.heads} query heads do not divide over {a.kv_heads} key / value heads")
        return a


@dataclass(frozen=True)
class LayerConfig:
    gla: GlaConfig
    attention: Optional[AttentionConfig] = None      # 'parallel' layers
    left_scale: float = 1.0
    right_scale: float = 1.0
    ff: int = 0                                      # 0: no feed-forward
    weights: int = 0                                 # the layer whose tensors it uses (its own index: its own)


@dataclass(frozen=True)
class TobovikConfig:
    vocab: int
    width: int
    eps: float
    layers: tuple = field(default_factory=tuple)

    @staticmethod
    def from_dict(cfg: dict) -> "TobovikConfig":
        entries, layers = cfg["layers"], []
        for i, entry in enumerate(entries):
            kind, m, mlp = entry["type"], entry["mixer"], entry.get("mlp")
            if kind == "gla":
                args = dict(gla=GlaConfig.from_dict(m))
            elif kind == "parallel":
                args = dict(gla=GlaConfig.from_dict(m["right"]), attention=AttentionConfig.from_dict(m["left"]), left_scale=float(m["left_scale"]),
                            right_scale=float(m["right_scale"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer '{kind}'")
            if mlp:
                if mlp["kind"] != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
                args.update(ff=int(mlp["ff"]))
            owner, seen = i, set()
            while entries[owner].get("weights_of") is not None:
                seen.add(owner)
                owner = int(entries[owner]["weights_of"])
                if not 0 <= owner < len(entries) or owner in seen:
                    raise ValueError(f"layer {i}: weights_of leads to no layer with weights of its own")
            layers.append(LayerConfig(weights=owner, **args))
        for i, layer in enumerate(layers):
            src = layers[layer.weights]
            if (src.gla, src.attention, src.ff) != (layer.gla, layer.attention, layer.ff):
                raise ValueError(f"layer {i}: sizes differ from those of layer {layer.weights}, whose weights it uses")
        return TobovikConfig(int(cfg["vocab"]), int(cfg["width"]), float(cfg["norm"]["eps"]), tuple(layers))


def gla_prefixes(cfg: TobovikConfig):
    """Tensor prefix of every gated-linear-attention mixer that has weights of its own."""
    return [f"l{i}.mix" + (".right" if layer.attention else "") for i, layer in enumerate(cfg.layers) if layer.weights == i]


class Tobovik(RowModel):
    def _operand_of(self, x):
        """The residual stream as operand of linear layers."""
        return self.graph.cast(x, FMT_BF16) if self._operand == FMT_BF16 else x

    def _build(self, g: Graph) -> int:
        cfg, op, eps = self.cfg, self._operand, self.cfg.eps
        x = g.embedding_positions(self.token_ids, self._mat("embed", cfg.vocab, cfg.width), self.pos, 1.0, POSITION_BASE)
        for i, layer in enumerate(cfg.layers):
            p = f"l{layer.weights}"
            h = self._operand_of(x)
            if layer.attention:
                y = self._parallel(g, i, f"{p}.mix", layer, h)
            else:
                inputs = self._gla_inputs(f"{p}.mix", layer.gla, h)
                y = self._linear(self._gla(g, i, f"{p}.mix", layer.gla, inputs), f"{p}.mix.o", cfg.width, layer.gla.heads * layer.gla.vdim)
            x = g.add(x, g.norm(y, self._vec(f"{p}.norm1", cfg.width), eps))
            if layer.ff:
                f, h = f"{p}.mlp", self._operand_of(x)
                y = g.silu_glu(self._linear(h, f"{f}.gate", layer.ff, cfg.width), self._linear(h, f"{f}.up", layer.ff, cfg.width), op)
                x = g.add(x, g.norm(self._linear(y, f"{f}.down", cfg.width, layer.ff), self._vec(f"{p}.norm2", cfg.width), eps))
            self._taps.append(x)
        h = g.norm(g.pick_rows(x, self.picked), self._vec("final.norm", cfg.width), eps, 0.0, op)
        return self._linear(h, "head", cfg.vocab, cfg.width)

    def _parallel(self, g, i, p, layer, h):
        a, width = layer.attention, self.cfg.width
        # the projections of both mixers first: layers of one input next to each other run as one launch
        q = self._linear(h, f"{p}.left.q", a.heads * a.dim, width, f"{p}.left.q.b")
        k = self._linear(h, f"{p}.left.k", a.kv_heads * a.dim, width, f"{p}.left.k.b")
        v = self._linear(h, f"{p}.left.v", a.kv_heads * a.vdim, width, f"{p}.left.v.b")
        gate = self._linear(h, f"{p}.left.g", a.heads * a.vdim, width)
        inputs = self._gla_inputs(f"{p}.right", layer.gla, h)
        left = self._attention(g, i, f"{p}.left", a, q, k, v, gate)
        right = self._gla(g, i, f"{p}.right", layer.gla, inputs)
        left = self._linear(left, f"{p}.left.o", width, a.heads * a.vdim)
        right = self._linear(right, f"{p}.right.o", width, layer.gla.heads * layer.gla.vdim)
        return g.scaled_sum(left, right, layer.left_scale, layer.right_scale)

    def _attention(self, g, i, p, a, q, k, v, gate):
        cfg = self.cfg
        cache = g.parameter_f16 if self._operand == FMT_BF16 else g.parameter
        keys = cache(f"l{i}.key_cache", [self.max_tokens, a.kv_heads * a.dim])
        values = cache(f"l{i}.value_cache", [self.max_tokens, a.kv_heads * a.vdim])
        q = g.norm(q, self._vec(f"{p}.q.norm", a.heads * a.dim), cfg.eps)
        k = g.norm(k, self._vec(f"{p}.k.norm", a.kv_heads * a.dim), cfg.eps)
        q = g.query_temperature(q, self.pos, a.temp_coef, a.temp_every)
        keys, values = g.cache_append(k, keys, self.pos), g.cache_append(v, values, self.pos)
        o = g.attention(q, keys, values, self.pos, a.heads, a.kv_heads, a.dim, a.vdim, a.scale)
        return g.head_gate(o, gate, a.heads, act=GATE_SIGMOID, out_dtype=self._operand)

    def _gla_inputs(self, p, m, h):
        width, rank = self.cfg.width, self.lora_rank[p]
        return tuple(self._linear(h, f"{p}.{s}", n, width) for s, n in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim),
                                                                          ("g", m.heads * m.vdim), ("a1", rank)))

    def _gla(self, g, i, p, m, inputs):
        q, k, v, gate, low = inputs
        n = m.heads * m.dim
        decay = g.lora_sigmoid_decay(low, self._mat(f"{p}.a2", n, self.lora_rank[p]), self._vec(f"{p}.a2.b", n), m.tau)
        state = g.parameter(f"l{i}.gla_state", [lib.mgq_gla_state_elements(m.heads, m.dim, m.vdim)])
        o = g.gla(q, k, v, decay, state, m.heads, self._operand)
        return g.head_gate(o, gate, m.heads, self._vec(f"{p}.norm", m.vdim), self.cfg.eps, GATE_SILU, self._operand)

    @staticmethod
    def from_tensors(config: dict, tensors, **kw) -> "Tobovik":
        cfg = TobovikConfig.from_dict(config)
        model = Tobovik(cfg, lora_rank={p: tensors.shape(f"{p}.a1")[0] for p in gla_prefixes(cfg)}, **kw)
        model.load(tensors)
        return model
