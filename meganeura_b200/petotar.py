"""Petotar: a decoder whose layers mix RWKV-style time mixing ('wkv'), mLSTM matrix memories
('mlstm') and latent attention over a sliding window ('latent_attention'), each followed by an
optional clamped GLU.  Built from Graph operators; the session runs whole prompts, portions and
single tokens from the same graph (row-dynamic inputs).

Every size and constant comes from config.json or a tensor's shape.  Weights stay bf16 on the
device; with dtype float32 the activations, caches and matrix products are f32, with bfloat16 the
operands of the linear layers and the latent cache are bf16 (norms, gates, decays, recurrent state,
attention scores and the residual stream are f32 in both).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

from ._lib import FMT_BF16, GATE_SIGMOID, GATE_SILU, lib
from .graph import Graph
from .row_model import RowModel

GLU_ALPHA = 1.702            # fixed by the design
SHIFTS = "rkvgw"             # token-shift mixes of a wkv layer, in slot order
MIXERS = ("wkv", "mlstm", "latent_attention")


@dataclass(frozen=True)
class LayerConfig:
    type: str
    heads: int
    dim: int                             # query / key dimensions of a head (latent attention: the unrotated ones)
    vdim: int
    gate_cap: float = 0.0                # mlstm
    kv_rank: int = 0                     # latent attention from here on
    rot_dim: int = 0
    rot_base: float = 1.0
    scale: float = 1.0
    window: int = 0
    kv_from: Optional[int] = None
    ff: int = 0                          # 0: no feed-forward
    limit: float = 0.0


@dataclass(frozen=True)
class PetotarConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    layers: tuple = field(default_factory=tuple)

    @staticmethod
    def from_dict(cfg: dict) -> "PetotarConfig":
        layers = []
        for i, entry in enumerate(cfg["layers"]):
            kind, m, mlp = entry["type"], entry["mixer"], entry.get("mlp")
            if kind not in MIXERS:
                raise ValueError(f"layer {i}: unknown mixer '{kind}'")
            args = dict(type=kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m.get("vdim", m["dim"])))
            if kind == "mlstm":
                args["gate_cap"] = float(m["gate_cap"])
            if kind == "latent_attention":
                rot = m["rot"]
                if int(rot["dims"]) != int(m["rot_dim"]):
                    raise ValueError(f"layer {i}: rot.dims {rot['dims']} differs from rot_dim {m['rot_dim']}")
                args.update(kv_rank=int(m["kv_rank"]), rot_dim=int(m["rot_dim"]), rot_base=float(rot["base"]), scale=float(m["scale"]),
                            window=int(m["mask"]["size"]), kv_from=None if m.get("kv_from") is None else int(m["kv_from"]))
            if mlp:
                if mlp["kind"] != "dense":
                    raise ValueError(f"layer {i}: unknown feed-forward '{mlp['kind']}'")
                args.update(ff=int(mlp["ff"]), limit=float(mlp["limit"]))
            layers.append(LayerConfig(**args))
        for i, layer in enumerate(layers):
            if layer.kv_from is None:
                continue
            j = layer.kv_from
            if not 0 <= j < i or layers[j].type != "latent_attention" or layers[j].kv_from is not None:
                raise ValueError(f"layer {i}: kv_from {j} is not an earlier latent-attention layer with a cache of its own")
            src = layers[j]
            if (src.kv_rank, src.rot_dim, src.rot_base) != (layer.kv_rank, layer.rot_dim, layer.rot_base):
                raise ValueError(f"layer {i}: latent or rotation differs from layer {j}, whose cache it reads")
        return PetotarConfig(int(cfg["vocab"]), int(cfg["width"]), float(cfg["norm"]["eps"]), float(cfg["embedding"]["scale"]), tuple(layers))


class Petotar(RowModel):
    """max_tokens bounds the latent caches together with the windows."""

    # ---- graph
    def _window(self, layer):
        return min(layer.window, self.max_tokens)

    def _build(self, g: Graph) -> int:
        cfg, op = self.cfg, self._operand
        embed = self._mat("embed", cfg.vocab, cfg.width)
        x = g.embedding_scaled(self.token_ids, embed, cfg.embedding_scale)
        caches = {}
        for i, layer in enumerate(cfg.layers):
            norm1 = self._vec(f"l{i}.norm1", cfg.width)
            mixer = {"wkv": self._wkv, "mlstm": self._mlstm, "latent_attention": self._latent}[layer.type]
            x = g.add(x, mixer(g, i, layer, x, norm1, caches))
            if layer.ff:
                f = f"l{i}.mlp"
                h = g.norm(x, self._vec(f"l{i}.norm2", cfg.width), cfg.eps, 1.0, op)
                gate = g.bias_add(self._linear(h, f"{f}.gate", layer.ff, cfg.width), self._vec(f"{f}.gate.b", layer.ff))
                up = g.bias_add(self._linear(h, f"{f}.up", layer.ff, cfg.width), self._vec(f"{f}.up.b", layer.ff))
                y = g.clamped_glu(gate, up, layer.limit, GLU_ALPHA, op)
                x = g.add(x, g.bias_add(self._linear(y, f"{f}.down", cfg.width, layer.ff), self._vec(f"{f}.down.b", cfg.width)))
            self._taps.append(x)
        h = g.norm(g.pick_rows(x, self.picked), self._vec("final.norm", cfg.width), cfg.eps, 1.0, op)
        return g.matmul_bt(h, embed)

    def _wkv(self, g, i, layer, x, norm1, _):
        cfg, p, n = self.cfg, f"l{i}.mix", layer.heads * layer.dim
        rank = self.lora_rank[i]
        shift = g.parameter(f"{p}.shift_state", [2, cfg.width])
        mus = [self._vec(f"{p}.mu.{s}", cfg.width) for s in SHIFTS]
        mixes = g.token_shift(g.norm(x, norm1, cfg.eps, 1.0), mus, shift, self._operand)
        r, k, v, gate = (self._linear(g.slot(mixes, j), f"{p}.{s}", n, cfg.width) for j, s in enumerate("rkvg"))
        low = self._linear(g.slot(mixes, 4), f"{p}.w1", rank, cfg.width)
        decay = g.lora_decay(low, self._mat(f"{p}.w2", n, rank), self._vec(f"{p}.w0", n))
        state = g.parameter(f"{p}.state", [lib.mgq_wkv_state_elements(layer.heads, layer.dim)])
        o = g.wkv(r, k, v, decay, self._vec(f"{p}.u", n), state, layer.heads, shift)
        o = g.head_gate(o, gate, layer.heads, self._vec(f"{p}.norm", n), cfg.eps, GATE_SILU, self._operand)
        return self._linear(o, f"{p}.o", cfg.width, n)

    def _mlstm(self, g, i, layer, x, norm1, _):
        cfg, p, n, nv = self.cfg, f"l{i}.mix", layer.heads * layer.dim, layer.heads * layer.vdim
        h = g.norm(x, norm1, cfg.eps, 1.0, self._operand)
        q, k = self._linear(h, f"{p}.q", n, cfg.width), self._linear(h, f"{p}.k", n, cfg.width)
        v, gate = self._linear(h, f"{p}.v", nv, cfg.width), self._linear(h, f"{p}.g", nv, cfg.width)
        gi = g.bias_add(self._linear(h, f"{p}.i", layer.heads, cfg.width), self._vec(f"{p}.i.b", layer.heads))
        gf = g.bias_add(self._linear(h, f"{p}.f", layer.heads, cfg.width), self._vec(f"{p}.f.b", layer.heads))
        state = g.parameter(f"{p}.state", [lib.mgq_mlstm_state_elements(layer.heads, layer.dim, layer.vdim)])
        o = g.mlstm(q, k, v, gi, gf, state, layer.heads, layer.gate_cap)
        o = g.head_gate(o, gate, layer.heads, self._vec(f"{p}.norm", nv), cfg.eps, GATE_SIGMOID, self._operand)
        return self._linear(o, f"{p}.o", cfg.width, nv)

    def _latent(self, g, i, layer, x, norm1, caches):
        cfg, p = self.cfg, f"l{i}.mix"
        row = layer.kv_rank + layer.rot_dim
        h = g.norm(x, norm1, cfg.eps, 1.0, self._operand)
        q = self._linear(h, f"{p}.q", layer.heads * (layer.dim + layer.rot_dim), cfg.width)
        gate = self._linear(h, f"{p}.g", layer.heads * layer.vdim, cfg.width)
        if layer.kv_from is None:
            # a ring: the widest window of the layers that read it, in front of the step's own rows
            readers = [self._window(b) for j, b in enumerate(cfg.layers) if j == i or b.kv_from == i]
            slots = max(readers) - 1 + self.max_rows
            cache = (g.parameter_bf16 if self._operand == FMT_BF16 else g.parameter)(f"{p}.latent_cache", [slots, row])
            down = self._linear(h, f"{p}.dkv", row, cfg.width)
            caches[i] = g.latent_cache_write(down, self._vec(f"{p}.dkv.norm", layer.kv_rank), cache, self.pos, layer.rot_dim, layer.rot_base, cfg.eps)
        cache = caches[i if layer.kv_from is None else layer.kv_from]
        uk = self._mat(f"{p}.uk", layer.heads * layer.dim, layer.kv_rank)
        uv = self._mat(f"{p}.uv", layer.heads * layer.vdim, layer.kv_rank)
        o = g.latent_attention(q, cache, uk, uv, self.pos, layer.heads, layer.dim, layer.rot_dim, layer.vdim, self._window(layer), layer.scale,
                               layer.rot_base)
        o = g.head_gate(o, gate, layer.heads, act=GATE_SIGMOID, out_dtype=self._operand)
        return self._linear(o, f"{p}.o", cfg.width, layer.heads * layer.vdim)

    @staticmethod
    def from_tensors(config: dict, tensors, **kw) -> "Petotar":
        cfg = PetotarConfig.from_dict(config)
        ranks = {i: tensors.shape(f"l{i}.mix.w1")[0] for i, layer in enumerate(cfg.layers) if layer.type == "wkv"}
        model = Petotar(cfg, lora_rank=ranks, **kw)
        model.load(tensors)
        return model
