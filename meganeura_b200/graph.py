"""Graph / build_inference_session / Session with meganeura's names, over the C ABI.

The graph, the plan and the session live in C++ (csrc/mgq_session.cpp); this module only holds
handles.  Method names and argument meaning follow meganeura (src/graph.rs:714-795,
src/train.rs:380-389, src/runtime.rs:2327-2345, 2612-2643, 2786-2791, 2835-2959) so tests read
like the reference's (tests/gemv_parity.rs, tests/gpu_smoke.rs:2680-2771).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from enum import IntEnum

import numpy as np

from ._lib import FMT_F32, GATE_SIGMOID, check, last_error, lib, MgqError


class ShaderEntry(IntEnum):
    MatMul = 0
    FusedMatMulAdd = 1
    MatMulGemv = 2
    MatMulGemvAdd = 3
    Add = 4
    Embedding = 5
    RmsNorm = 6
    RoPEDynamic = 7
    CacheWrite = 8
    CachedAttention = 9
    SwiGLU = 10
    SwiGLUConcat = 11
    RoPECacheWrite = 12
    AllGather = 13
    MatMulGemvBT = 14
    Linear = 15
    LinearGLU = 16
    BiasAdd = 17
    PickRows = 18
    Norm = 19
    TokenShift = 20
    Decay = 21
    Wkv = 22
    Mlstm = 23
    HeadGate = 24
    LatentCacheWrite = 25
    LatentAttention = 26
    ClampedGLU = 27
    Cast = 28
    ScaledSum = 29
    ResidualNorm = 30
    Gla = 31
    QueryTemperature = 32
    CacheAppend = 33
    Attention = 34
    AttentionInputs = 35


class WeightFormat(IntEnum):
    F32 = 0
    F16 = 1
    Q4 = 2
    Q8 = 3
    BF16 = 4


@dataclass
class Dispatch:
    shader: ShaderEntry
    workgroups: tuple
    params: tuple
    weight_format: WeightFormat
    label: str


@dataclass
class ExecutionPlan:
    dispatches: list


def _shape(shape):
    arr = (ctypes.c_size_t * len(shape))(*[int(s) for s in shape])
    return arr, len(shape)


def _node(rc: int) -> int:
    if rc < 0:
        raise MgqError(-rc, last_error())
    return rc


class Graph:
    def __init__(self):
        self._h = lib.mgq_graph_new()

    def __del__(self):
        if getattr(self, "_h", None):
            lib.mgq_graph_free(self._h)
            self._h = None

    def input(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_input(self._h, name.encode(), *_shape(shape)))

    def parameter(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_parameter(self._h, name.encode(), *_shape(shape)))

    def parameter_q4(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_parameter_q4(self._h, name.encode(), *_shape(shape)))

    def parameter_q8(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_parameter_q8(self._h, name.encode(), *_shape(shape)))

    def parameter_f16(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_parameter_f16(self._h, name.encode(), *_shape(shape)))

    def matmul(self, a: int, b: int) -> int:
        return _node(lib.mgq_graph_matmul(self._h, a, b))

    def add(self, a: int, b: int) -> int:
        return _node(lib.mgq_graph_add(self._h, a, b))

    def input_u32(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_input_u32(self._h, name.encode(), *_shape(shape)))

    def embedding(self, indices: int, table: int) -> int:
        return _node(lib.mgq_graph_embedding(self._h, indices, table))

    def rms_norm(self, x: int, weight: int, eps: float) -> int:
        return _node(lib.mgq_graph_rms_norm(self._h, x, weight, eps))

    def rope_dynamic_offset(self, x: int, theta: float, offset_input: int, head_dim: int) -> int:
        return _node(lib.mgq_graph_rope_dynamic_offset(self._h, x, theta, offset_input, head_dim))

    def cache_write(self, new_kv: int, cache: int, kv_pos: int) -> int:
        return _node(lib.mgq_graph_cache_write(self._h, new_kv, cache, kv_pos))

    def cached_attention(self, q: int, k_cache: int, v_cache: int, kv_pos: int, num_heads: int, num_kv_heads: int,
                         head_dim: int) -> int:
        return _node(lib.mgq_graph_cached_attention(self._h, q, k_cache, v_cache, kv_pos, num_heads, num_kv_heads, head_dim))

    def swiglu(self, gate: int, up: int) -> int:
        return _node(lib.mgq_graph_swiglu(self._h, gate, up))

    def swiglu_concat(self, x: int) -> int:
        return _node(lib.mgq_graph_swiglu_concat(self._h, x))

    def matmul_bt(self, a: int, b: int) -> int:
        """Graph::matmul_bt (src/graph.rs:809-817): a [M, K] @ b[N, K]^T, b an f32 parameter."""
        return _node(lib.mgq_graph_matmul_bt(self._h, a, b))

    # ---- row-dynamic graphs and the operators of recurrent / attention decoders (mgq.h)
    def input_u32_rows(self, name: str, capacity: int, which: int) -> int:
        """u32 input of up to `capacity` rows; Session.set_rows(which, n) sets the count of a step."""
        return _node(lib.mgq_graph_input_u32_rows(self._h, name.encode(), capacity, which))

    def parameter_bf16(self, name: str, shape) -> int:
        return _node(lib.mgq_graph_parameter_bf16(self._h, name.encode(), *_shape(shape)))

    def embedding_scaled(self, indices: int, table: int, scale: float) -> int:
        return _node(lib.mgq_graph_embedding_scaled(self._h, indices, table, scale))

    def embedding_positions(self, indices: int, table: int, pos: int, scale: float = 1.0, base: float = 10000.0) -> int:
        """embedding_scaled plus the sinusoidal vector of every token's position (pos: position of row 0)."""
        return _node(lib.mgq_graph_embedding_positions(self._h, indices, table, pos, scale, base))

    def cast(self, x: int, out_dtype: int) -> int:
        return _node(lib.mgq_graph_cast(self._h, x, out_dtype))

    def scaled_sum(self, a: int, b: int, sa: float, sb: float) -> int:
        return _node(lib.mgq_graph_scaled_sum(self._h, a, b, sa, sb))

    def pick_rows(self, x: int, index: int) -> int:
        return _node(lib.mgq_graph_pick_rows(self._h, x, index))

    def norm(self, x: int, weight: int, eps: float, weight_offset: float = 0.0, out_dtype: int = FMT_F32) -> int:
        return _node(lib.mgq_graph_norm(self._h, x, weight, eps, weight_offset, out_dtype))

    def bias_add(self, x: int, bias: int) -> int:
        return _node(lib.mgq_graph_bias_add(self._h, x, bias))

    def clamped_glu(self, gate: int, up: int, limit: float, alpha: float, out_dtype: int = FMT_F32) -> int:
        return _node(lib.mgq_graph_clamped_glu(self._h, gate, up, limit, alpha, out_dtype))

    def silu_glu(self, gate: int, up: int, out_dtype: int = FMT_F32) -> int:
        return _node(lib.mgq_graph_silu_glu(self._h, gate, up, out_dtype))

    def token_shift(self, h: int, mu, state: int, out_dtype: int = FMT_F32) -> int:
        """[len(mu), rows, width] mixes of every token with the one before it; take one with slot()."""
        arr = (ctypes.c_int * len(mu))(*mu)
        return _node(lib.mgq_graph_token_shift(self._h, h, arr, len(mu), state, out_dtype))

    def slot(self, x: int, index: int) -> int:
        return _node(lib.mgq_graph_slot(self._h, x, index))

    def lora_decay(self, low: int, w2: int, w0: int) -> int:
        return _node(lib.mgq_graph_lora_decay(self._h, low, w2, w0))

    def lora_sigmoid_decay(self, low: int, w2: int, bias: int, tau: float) -> int:
        return _node(lib.mgq_graph_lora_sigmoid_decay(self._h, low, w2, bias, tau))

    def gla(self, q: int, k: int, v: int, decay: int, state: int, heads: int, product_dtype: int = FMT_F32) -> int:
        return _node(lib.mgq_graph_gla(self._h, q, k, v, decay, state, heads, product_dtype))

    def query_temperature(self, x: int, pos: int, coef: float, every: float) -> int:
        return _node(lib.mgq_graph_query_temperature(self._h, x, pos, coef, every))

    def cache_append(self, x: int, cache: int, pos: int) -> int:
        return _node(lib.mgq_graph_cache_append(self._h, x, cache, pos))

    def attention(self, q: int, k_cache: int, v_cache: int, pos: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float) -> int:
        return _node(lib.mgq_graph_attention(self._h, q, k_cache, v_cache, pos, heads, kv_heads, dim, vdim, scale))

    def wkv(self, r: int, k: int, v: int, decay: int, u: int, state: int, heads: int, shift_state: int = -1) -> int:
        return _node(lib.mgq_graph_wkv(self._h, r, k, v, decay, u, state, shift_state, heads))

    def mlstm(self, q: int, k: int, v: int, gate_i: int, gate_f: int, state: int, heads: int, gate_cap: float) -> int:
        return _node(lib.mgq_graph_mlstm(self._h, q, k, v, gate_i, gate_f, state, heads, gate_cap))

    def head_gate(self, o: int, gate: int, heads: int, weight: int = -1, eps: float = 0.0, act: int = GATE_SIGMOID,
                  out_dtype: int = FMT_F32) -> int:
        return _node(lib.mgq_graph_head_gate(self._h, o, weight, gate, heads, eps, act, out_dtype))

    def latent_cache_write(self, down: int, weight: int, cache: int, pos: int, rot_dim: int, rot_base: float, eps: float) -> int:
        return _node(lib.mgq_graph_latent_cache_write(self._h, down, weight, cache, pos, rot_dim, rot_base, eps))

    def latent_attention(self, q: int, cache: int, uk: int, uv: int, pos: int, heads: int, dim: int, rot_dim: int, vdim: int, window: int,
                         scale: float, rot_base: float) -> int:
        return _node(lib.mgq_graph_latent_attention(self._h, q, cache, uk, uv, pos, heads, dim, rot_dim, vdim, window, scale, rot_base))

    def all_gather(self, x: int, world: int) -> int:
        """This rank's [1, n] slice -> the whole [1, n * world] vector, rank-major (column-sharded
        models; no reference counterpart: the reference is single-device)."""
        return _node(lib.mgq_graph_all_gather(self._h, x, world))

    def slice_columns(self, x: int, first: int, count: int) -> int:
        """Columns [first, first + count) of a [1, n] node, as a view."""
        return _node(lib.mgq_graph_slice_columns(self._h, x, first, count))

    def set_outputs(self, ids) -> None:
        arr = (ctypes.c_int * len(ids))(*ids)
        check(lib.mgq_graph_set_outputs(self._h, arr, len(ids)))


class Session:
    def __init__(self, handle):
        self._h = handle

    def __del__(self):
        if getattr(self, "_h", None):
            lib.mgq_session_free(self._h)
            self._h = None

    def set_parameter(self, name: str, data) -> None:
        data = np.ascontiguousarray(data, dtype=np.float32).reshape(-1)
        check(lib.mgq_session_set_parameter(self._h, name.encode(), data.ctypes.data, data.size))

    def upload_param(self, name: str, raw) -> None:
        raw = np.ascontiguousarray(raw).view(np.uint8).reshape(-1)
        check(lib.mgq_session_upload_param(self._h, name.encode(), raw.ctypes.data, raw.size))

    def set_input(self, name: str, data) -> None:
        data = np.ascontiguousarray(data, dtype=np.float32).reshape(-1)
        check(lib.mgq_session_set_input(self._h, name.encode(), data.ctypes.data, data.size))

    def save_checkpoint(self, path) -> None:
        check(lib.mgq_session_save_checkpoint(self._h, str(path).encode()))

    def load_checkpoint(self, path) -> None:
        check(lib.mgq_session_load_checkpoint(self._h, str(path).encode()))

    def set_input_u32(self, name: str, data) -> None:
        data = np.ascontiguousarray(data, dtype=np.uint32).reshape(-1)
        check(lib.mgq_session_set_input_u32(self._h, name.encode(), data.ctypes.data, data.size))

    def set_rows(self, which: int, count: int) -> None:
        """Row-dynamic sessions: rows of the following steps (ROWS_TOKENS or ROWS_PICKED)."""
        check(lib.mgq_session_set_rows(self._h, which, count))

    def reset_state(self) -> None:
        """Clear every recurrent state and latent cache (the next step starts a new sequence)."""
        check(lib.mgq_session_reset_state(self._h))

    def step(self) -> None:
        check(lib.mgq_session_step(self._h))

    def capture(self) -> None:
        """Capture the dispatch list into a CUDA graph (after at least one ordinary step)."""
        check(lib.mgq_session_capture(self._h))

    def enable_greedy(self, output_index: int, token_input: str, pos_input: str, history_cap: int) -> None:
        """Pick the next token on the device after every step and feed it (and position + 1) back."""
        check(lib.mgq_session_enable_greedy(self._h, output_index, token_input.encode(), pos_input.encode(), history_cap))

    def read_tokens(self, first_pos: int, count: int) -> np.ndarray:
        out = np.empty(count, dtype=np.uint32)
        check(lib.mgq_session_read_tokens(self._h, first_pos, out.ctypes.data, count))
        return out

    def wait(self) -> None:
        check(lib.mgq_session_wait(self._h))

    def read_output(self, length: int) -> np.ndarray:
        out = np.empty(length, dtype=np.float32)
        check(lib.mgq_session_read_output(self._h, out.ctypes.data, length))
        return out

    def read_output_by_index(self, index: int, length: int) -> np.ndarray:
        out = np.empty(length, dtype=np.float32)
        check(lib.mgq_session_read_output_by_index(self._h, index, out.ctypes.data, length))
        return out

    def plan(self) -> ExecutionPlan:
        count = lib.mgq_session_num_dispatches(self._h)
        dispatches = []
        for i in range(count):
            shader, wf = ctypes.c_int(), ctypes.c_int()
            wg, pr = (ctypes.c_uint32 * 3)(), (ctypes.c_uint32 * 4)()
            label = ctypes.create_string_buffer(128)
            check(lib.mgq_session_dispatch_info(self._h, i, ctypes.byref(shader), wg, pr, ctypes.byref(wf), label, 128))
            dispatches.append(Dispatch(ShaderEntry(shader.value), tuple(wg), tuple(pr), WeightFormat(wf.value), label.value.decode()))
        return ExecutionPlan(dispatches)

    def launch_count(self) -> int:
        return int(lib.mgq_session_launch_count(self._h))

    def set_profiling(self, enabled: bool) -> None:
        """Session::set_profiling: the next steps run one timed dispatch at a time (no graph replay)."""
        check(lib.mgq_session_set_profiling(self._h, 1 if enabled else 0))

    def gpu_timings(self):
        """Microseconds of every dispatch of the last profiled step."""
        import numpy as np
        n = int(lib.mgq_session_num_dispatches(self._h))
        out = np.zeros(n, dtype=np.float32)
        check(lib.mgq_session_gpu_timings(self._h, out.ctypes.data, n))
        return out

    def dump_gpu_timings(self) -> str:
        """Session::dump_gpu_timings: per-label totals of the last profiled step, largest first."""
        buf = ctypes.create_string_buffer(16384)
        check(lib.mgq_session_dump_gpu_timings(self._h, buf, len(buf)))
        return buf.value.decode()

    def num_groups(self) -> int:
        """Session::num_groups: barrier groups of the dispatch list."""
        n = int(lib.mgq_session_num_groups(self._h))
        if n < 0:
            check(-n)
        return n

    # ---- column-sharded sessions (graphs with all_gather nodes)
    def exchange_slices(self):
        """Floats this rank contributes to each all_gather, in execution order."""
        n = int(lib.mgq_session_num_exchanges(self._h))
        if n < 0:
            check(-n)
        out = []
        for i in range(n):
            slice_len, world = ctypes.c_uint32(), ctypes.c_uint32()
            check(lib.mgq_session_exchange_info(self._h, i, ctypes.byref(slice_len), ctypes.byref(world)))
            out.append(int(slice_len.value))
        return out

    def bind_exchanges(self, exchange) -> None:
        """Binds every all_gather to a PeerExchange built from exchange_slices() (kept alive here)."""
        for i in range(len(exchange.gather_sizes)):
            check(lib.mgq_session_bind_exchange(self._h, i, exchange.push_ptr(i), exchange.vec_ptr(i)))
        check(lib.mgq_session_bind_exchange_state(self._h, exchange.epoch_ptr, exchange.error_ptr, exchange.local + exchange.off_blocks))
        self._exchange = exchange

    def check_exchange(self) -> None:
        check(lib.mgq_session_check_exchange(self._h))


def build_inference_session(graph: Graph) -> Session:
    handle = ctypes.c_void_p()
    check(lib.mgq_build_inference_session(graph._h, ctypes.byref(handle)))
    return Session(handle)
