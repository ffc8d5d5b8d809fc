"""The engine's kernels as Python calls over torch tensors (ctypes into the built libraries).

There is no fallback: if a library cannot be built or loaded, or a kernel
refuses a size, the call raises. Calls launch on torch's current stream.
"""
from __future__ import annotations

import bisect
import ctypes
import os
from typing import Dict, Optional

import numpy as np
import torch

from . import build

_DT = {torch.float32: 0, torch.bfloat16: 1}

_ERRORS = {
    -1: "unsupported dtype",
    -2: "a size the kernel refuses",
    -3: "a pointer or stride is not aligned as the kernel needs",
    -4: "a size beyond the kernel's stated maximum",
}


class KernelError(RuntimeError):
    pass


def _check(rc: int, what: str) -> None:
    if rc == 0:
        return
    if rc in _ERRORS:
        raise KernelError(f"{what}: {_ERRORS[rc]}")
    if rc < 0:
        raise KernelError(f"{what}: library error {rc}")
    raise KernelError(f"{what}: CUDA error {rc} at launch")


def _p(t: Optional[torch.Tensor]):
    return ctypes.c_void_p(t.data_ptr() if t is not None else 0)


def _stream():
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


class _PinnedStream:
    """While active, the kernels launch on the given stream handle without asking torch for the current stream at
    every launch (that question costs several microseconds, a hundred times a step)."""

    def __init__(self, kernels, handle):
        self.kernels, self.handle, self.before = kernels, handle, None

    def __enter__(self):
        self.before = self.kernels._stream_handle
        self.kernels._stream_handle = ctypes.c_void_p(self.handle) if self.handle is not None else None
        return self

    def __exit__(self, *exc):
        self.kernels._stream_handle = self.before
        return False


def core_jobs():
    return [
        {"name": "sb_core", "sources": ["elementwise.cu", "skinny_linear.cu", "gemm_tcgen05.cu"]},
        {"name": "sb_gemm", "sources": ["gemm_cublas.cu"], "libs": ["cublas"]},
    ]


def sequence_job():
    """Kernels of the mixers with recurrent state (built when a model first asks for them)."""
    return {"name": "sb_seq", "sources": ["sequence_ops.cu", "chunked_retention.cu"]}


def experts_job():
    """Kernels of feed-forwards made of experts (built when a model first asks for them)."""
    return {"name": "sb_moe", "sources": ["routed_experts.cu"]}


def projection_job():
    """Layer norm, grouped norm, whole-projection query/key norm with temperature, latent-attention preparation, activations."""
    return {"name": "sb_prep", "sources": ["projection_ops.cu", "grouped_norm.cu"]}


def attention_job(head_dim: int):
    return {"name": f"sb_attention_hd{head_dim}", "sources": ["attention_simt.cu", "attention_mma.cu", "attention_tc.cu"],
            "defines": [f"SB_HEAD_DIM={head_dim}"]}


def talking_attention_job(head_dim: int):
    """Attention whose heads' weights are mixed before the values (built when a model first asks for it)."""
    return {"name": f"sb_talk_hd{head_dim}", "sources": ["talking_attention.cu", "talking_attention_tc.cu"], "defines": [f"SB_HEAD_DIM={head_dim}"]}


def layer_run_job(head_dim: int):
    # SERVE_B200_STACK_DEFINES: extra -D settings for experiments with the kernel's constants (space separated)
    extra = os.environ.get("SERVE_B200_STACK_DEFINES", "").split()
    return {"name": f"sb_stack_hd{head_dim}", "sources": ["decode_stack.cu"], "defines": [f"SB_HEAD_DIM={head_dim}"] + extra}


SUPPORTED_HEAD_DIMS = tuple(range(16, 257, 16))
# head sizes for which the kernel that runs whole layers of a decoding step is built
LAYER_RUN_HEAD_DIMS = (64, 128)

# one layer as decode_stack.h lays it out (SbStackLayer)
_STACK_LAYER = np.dtype([("wqkv", "u8"), ("wo", "u8"), ("wgu", "u8"), ("wdown", "u8"), ("norm1", "u8"), ("norm2", "u8"),
                         ("inv_freq", "u8"), ("kc", "u8"), ("vc", "u8"), ("eps1", "f4"), ("eps2", "f4"), ("scale_log2", "f4"),
                         ("rot", "i4"), ("window", "i4"), ("norm_f32", "i4"), ("group", "i4"), ("num_pages", "i4"),
                         ("write_cache", "i4"), ("pad", "i4")])
_STACK_MAX_GROUPS = 4
_STACK_MAX_ROWS = 16


class LayerRunPlan:
    """A run of layers that one launch of the decode-stack kernel takes: the layers' table on the device and what
    every step needs to call the kernel."""

    def __init__(self, lib, table, keep, n_layers, hidden, heads, kv_heads, head_dim, inter, groups, page_size, blocks):
        self.lib, self.table, self.keep, self.n_layers = lib, table, keep, n_layers
        self.hidden, self.heads, self.kv_heads, self.head_dim, self.inter = hidden, heads, kv_heads, head_dim, inter
        self.groups, self.page_size, self.blocks = groups, page_size, blocks
        self.takes: Dict[int, bool] = {}


def all_jobs():
    """Every library the engine can ask for (the build check compiles them all)."""
    return (core_jobs() + [sequence_job(), experts_job(), projection_job()] + [attention_job(d) for d in SUPPORTED_HEAD_DIMS]
            + [talking_attention_job(d) for d in SUPPORTED_HEAD_DIMS]
            + [layer_run_job(d) for d in LAYER_RUN_HEAD_DIMS])


class CudaKernels:
    """Loads (building if needed) the libraries and exposes one method per kernel."""

    def __init__(self, device="cuda:0", head_dims=(), verbose: bool = True):
        self.device = torch.device(device)
        if self.device.type == "cuda" and torch.cuda.is_available():
            self.TARGET_BLOCKS = torch.cuda.get_device_properties(self.device).multi_processor_count
        jobs = core_jobs() + [attention_job(d) for d in sorted(set(head_dims))]
        for j in jobs:
            j["verbose"] = verbose
        paths = build.build_many(jobs)
        self.paths = dict(paths)
        self._core = ctypes.CDLL(paths["sb_core"])
        self._gemm = ctypes.CDLL(paths["sb_gemm"])
        self._attn: Dict[int, ctypes.CDLL] = {}
        for d in set(head_dims):
            self._attn[d] = ctypes.CDLL(paths[f"sb_attention_hd{d}"])
            self._attn[d].sb_attention_mma_scratch_bytes.restype = ctypes.c_longlong
        self._verbose = verbose
        self._errors: Optional[torch.Tensor] = None
        self.force_simt_attention = False   # tests: run bfloat16 through the plain-arithmetic kernel
        self.use_skinny_linear = True       # tests: False sends every product to the library
        self.use_tcgen05 = True             # tests: False keeps many-row products in the library
        self.fuse_rope = True               # tests: False runs the rotary kernel after the q/k/v product
        self.use_tcgen05_attention = True   # tests: False keeps prompt portions on the mma.sync kernel
        if os.environ.get("SERVE_B200_TCGEN05_PLAIN") == "1":     # measurements: plain products on the tiles too
            self.tcgen05_for_plain_products = True
        self._stream_handle = None           # set by on_current_stream(): the stream every launch goes to
        self._routes: Dict[tuple, int] = {}  # which product kernel takes a shape (asked of the libraries once)
        self._tc_attention_ok: Dict[tuple, bool] = {}
        self._split_scratch = None           # partial results of the split-key merge
        self._sample_work = None
        self._keep = []
        self._tickets = []                   # zeroed int32 buffers of the split-key merge (kept alive for graphs)
        self.launches = 0         # launches of this engine's own kernels
        self.library_calls = 0    # library matrix products
        # Small decoding steps can run all layers in ONE launch (csrc/decode_stack.cu). Measured on a B200 at the
        # Llama-3.2-1B shape it is slower than the chain of separate kernels (about 80 us a layer against 42), so it is
        # off unless asked for (tests, and SERVE_B200_LAYER_RUNS=1 for measurements).
        self.use_layer_runs = os.environ.get("SERVE_B200_LAYER_RUNS", "0") == "1"
        self._seq = None                     # the library of sequence_job(), loaded at first use
        self._moe = None                     # the library of experts_job(), loaded at first use
        self._prep = None                    # the library of projection_job(), loaded at first use
        self._talk: Dict[int, ctypes.CDLL] = {}     # libraries of talking_attention_job(), by head size
        self._stack: Dict[int, ctypes.CDLL] = {}
        self._stack_sync = None              # two counters of the layer-run kernel's grid barrier (zero between launches)
        self._stack_partials = None
        self.layer_runs = 0                  # launches of the layer-run kernel
        self.layer_run_timing = None         # profiles: an int64 tensor [layers * 10] that receives block 0's phase stamps

    # ---- stream -----------------------------------------------------------
    def on_current_stream(self):
        """Context manager: look torch's current stream up once and launch on it until the block ends.
        Enter it again after switching streams (graph capture does)."""
        return _PinnedStream(self, torch.cuda.current_stream(self.device).cuda_stream)

    def _s(self):
        h = self._stream_handle
        return h if h is not None else ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)

    # ---- checks -----------------------------------------------------------
    @staticmethod
    def check_attention_shape(heads: int, kv_heads: int, head_dim: int) -> None:
        if head_dim % 16 or not (16 <= head_dim <= 256):
            raise KernelError(f"head_dim {head_dim} is not supported: the attention kernels take multiples of 16 from 16 to 256")
        if heads % kv_heads:
            raise KernelError(f"heads {heads} is not a multiple of kv_heads {kv_heads}")
        if heads > 65535:
            raise KernelError("more than 65535 heads")

    def _attention_lib(self, head_dim: int):
        lib = self._attn.get(head_dim)
        if lib is None:
            self.check_attention_shape(1, 1, head_dim)
            job = attention_job(head_dim)
            job["verbose"] = self._verbose
            path = build.build_library(**job)
            self.paths[job["name"]] = path
            lib = self._attn[head_dim] = ctypes.CDLL(path)
            lib.sb_attention_mma_scratch_bytes.restype = ctypes.c_longlong
        return lib

    def _talk_lib(self, head_dim: int):
        lib = self._talk.get(head_dim)
        if lib is None:
            self.check_attention_shape(1, 1, head_dim)
            job = talking_attention_job(head_dim)
            job["verbose"] = self._verbose
            path = build.build_library(**job)
            self.paths[job["name"]] = path
            lib = self._talk[head_dim] = ctypes.CDLL(path)
        return lib

    def prepare(self, head_dims=(), libraries=(), talking_head_dims=()) -> None:
        """Build side by side, and load, what a model is going to call: attention libraries for ``head_dims``, those with mixed
        heads for ``talking_head_dims`` and the optional libraries named ("seq", "moe", "prep"). Without this each is built when
        first called."""
        named = {"seq": sequence_job, "moe": experts_job, "prep": projection_job}
        jobs = [attention_job(d) for d in sorted(set(head_dims)) if d not in self._attn]
        for d in list(head_dims) + list(talking_head_dims):
            self.check_attention_shape(1, 1, d)
        jobs += [talking_attention_job(d) for d in sorted(set(talking_head_dims)) if d not in self._talk]
        jobs += [named[n]() for n in sorted(set(libraries)) if getattr(self, "_" + n) is None]
        if not jobs:
            return
        for j in jobs:
            j["verbose"] = self._verbose
        self.paths.update(build.build_many(jobs))
        for d in head_dims:
            self._attention_lib(d)
        for d in talking_head_dims:
            self._talk_lib(d)
        for n in libraries:
            getattr(self, f"_{n}_lib")()

    def errors_tensor(self) -> torch.Tensor:
        if self._errors is None:
            # [0]: cache writes that met a missing page; [1]: a bounded wait inside a kernel ran out
            self._errors = torch.zeros(4, dtype=torch.int32, device=self.device)
        return self._errors

    # The tensor-memory product works in 128 x 256 tiles, one CTA per SM: with fewer tiles than this most SMs
    # would idle and the library's split-k kernels are the better choice.
    TCGEN05_MIN_TILES = 96
    # A product without an epilogue of its own (output and down projection) goes to the library at every row count above the
    # few-rows kernel's: measured on a B200 at the 1B shapes from 128 to 4,096 rows the library is the faster one (2,048
    # rows: 14.9 against 16.2 us and 47.5 against 52.3 us; 3,072 rows: 20.7 / 26.9 and 69.7 / 95.9), and a prompt step of
    # 2,048 / 4,096 / 8,192 tokens went from 4.48 / 8.94 / 23.3 to 4.31 / 8.46 / 20.9 ms. The tiles earn their place where
    # an epilogue is fused (gate/up + SwiGLU, q/k/v + rotation + cache write). True: plain products use the tiles too (tests).
    tcgen05_for_plain_products = False

    def _tcgen05_worthwhile(self, m: int, n_acc: int) -> bool:
        return self.use_tcgen05 and (-(-m // 128)) * (-(-n_acc // 256)) >= self.TCGEN05_MIN_TILES

    def _wait_flag(self):
        return ctypes.c_void_p(self.errors_tensor().data_ptr() + 4)

    def check_errors(self) -> None:
        """Raise if a kernel met a page id or block index outside its table (synchronises)."""
        if self._errors is not None:
            n, timeouts = self._errors[:2].tolist()
            if n or timeouts:
                self._errors.zero_()
                if self._stack_sync is not None:
                    self._stack_sync.zero_()     # a barrier that gave up leaves its counters as they were
                if timeouts:
                    raise KernelError("a wait on a copy or tensor-core barrier inside a kernel ran out; the step's results are not valid")
                raise KernelError(f"{n} cache writes met a missing page or a block index beyond the block table")

    # ---- kernels ----------------------------------------------------------
    def fetch_ints(self, host_pinned, dev, n: int) -> None:
        """dev[:n] = host_pinned[:n] (int32, n a multiple of 4), copied by a kernel that reads the pinned host buffer."""
        self.launches += 1
        _check(self._core.sb_fetch_ints(_p(host_pinned), _p(dev), n, self._s()), "fetch of the step's inputs")

    def embedding(self, tokens, table, out, last_token=None, scale: float = 1.0) -> None:
        """out[t] = table[tokens[t]] * scale; an id -(s+1) is replaced by last_token[s] (the token last sampled for slot s)."""
        self.launches += 1
        _check(self._core.sb_embedding(_p(tokens), _p(table), _p(out), tokens.shape[0], table.shape[1], table.shape[0],
                                       _DT[table.dtype], _p(last_token), last_token.shape[0] if last_token is not None else 0,
                                       ctypes.c_float(scale), self._s()), "embedding")

    def embedding_pair(self, ctx, table, pairs, state, buckets: int, mul_prev: int, mul_cur: int, out, scale: float = 1.0) -> None:
        """out[t] = table[token] * scale + pairs[row], row = (previous token * mul_prev + token * mul_cur) mod buckets, or
        ``buckets`` for a sequence's first token. ``state`` [slots, 1] float holds, as an integer's bits, the last token of
        every request's previous portion, and takes this portion's."""
        t = ctx.tokens.shape[0]
        work = torch.empty(2 * t, dtype=torch.int32, device=out.device)
        last = getattr(ctx, "last_token", None)
        self.launches += 2
        _check(self._prep_lib().sb_embedding_pair(
            _p(ctx.tokens), _p(ctx.positions), _p(ctx.token_row), _p(ctx.cu_q), _p(ctx.slots), _p(state),
            ctypes.c_longlong(state.stride(0)), _p(last), last.shape[0] if last is not None else 0, _p(table), _p(pairs), table.shape[0],
            table.shape[1], int(buckets), ctypes.c_longlong(mul_prev), ctypes.c_longlong(mul_cur), ctypes.c_float(scale), _p(work), _p(out), t,
            _DT[table.dtype], self._s()), "embedding with a pair table")

    def bias_round(self, sums, bias, out) -> None:
        """out = sums (float) + bias (float [cols] or None), rounded once to out's type; both may be column slices."""
        if sums.dtype != torch.float32 or sums.shape != out.shape or sums.stride(1) != 1 or out.stride(1) != 1:
            raise KernelError("bias_round: float sums and an output of their shape")
        self.launches += 1
        _check(self._prep_lib().sb_bias_round(_p(sums), sums.stride(0), _p(bias), _p(out), out.stride(0), sums.shape[0], sums.shape[1],
                                              _DT[out.dtype], self._s()), "bias")

    def sigmoid_gate(self, a, gate, out, scale: float = 1.0) -> None:
        """out = scale * a * sigmoid(gate): gate [T, g] with g dividing a's columns (one number for each run of columns), of a's type
        or float, or None. a, gate and out may be column slices, a and out the same buffer."""
        if a.shape != out.shape or a.dtype != out.dtype or a.stride(1) != 1 or out.stride(1) != 1 or (
                gate is not None and (gate.dtype not in (a.dtype, torch.float32) or gate.stride(1) != 1)):
            raise KernelError("sigmoid_gate: operands of one type (the gate may be float), contiguous along their rows")
        self.launches += 1
        _check(self._prep_lib().sb_sigmoid_gate(_p(a), a.stride(0), _p(gate), gate.stride(0) if gate is not None else 0,
                                                gate.shape[1] if gate is not None else 0, _p(out), out.stride(0), a.shape[0], a.shape[1],
                                                ctypes.c_float(scale), _DT[a.dtype], 1 if gate is not None and gate.dtype == torch.float32 else 0,
                                                self._s()), "sigmoid gate")

    def softcap(self, x, cap: float) -> None:
        """x (float, contiguous) <- cap * tanh(x / cap)."""
        if x.dtype != torch.float32 or not x.is_contiguous():
            raise KernelError("softcap: float, contiguous")
        self.launches += 1
        _check(self._prep_lib().sb_softcap(_p(x), ctypes.c_longlong(x.numel()), ctypes.c_float(cap), self._s()), "capped logits")

    def add_rmsnorm(self, x, delta, weight, eps, out) -> None:
        self.launches += 1
        _check(self._core.sb_add_rmsnorm(_p(x), _p(delta), _p(None), _p(weight), _DT[weight.dtype], _p(out), x.shape[0],
                                         x.shape[1], ctypes.c_float(eps), _DT[out.dtype], self._s()), "add_rmsnorm")

    def add2_rmsnorm(self, x, delta, delta2, rows, weight, eps, out) -> None:
        """As add_rmsnorm (``rows`` None) or add_rmsnorm_rows with two deltas: x += delta + delta2, each added in float."""
        self.launches += 1
        n = rows.shape[0] if rows is not None else x.shape[0]
        _check(self._core.sb_add2_rmsnorm(_p(x), _p(delta), _p(delta2), _p(rows), _p(weight), _DT[weight.dtype], _p(out), n, x.shape[1],
                                          ctypes.c_float(eps), _DT[out.dtype], self._s()), "add_rmsnorm with two deltas")

    def add_rmsnorm_rows(self, x, delta, rows, weight, eps, out) -> None:
        self.launches += 1
        _check(self._core.sb_add_rmsnorm(_p(x), _p(delta), _p(rows), _p(weight), _DT[weight.dtype], _p(out), rows.shape[0],
                                         x.shape[1], ctypes.c_float(eps), _DT[out.dtype], self._s()), "add_rmsnorm_rows")

    def add_layernorm(self, x, delta, weight, eps, out) -> None:
        """x += delta; out = (x - mean) / sqrt(var + eps) * weight, row by row (x float, updated in place)."""
        self.launches += 1
        _check(self._prep_lib().sb_add_layernorm(_p(x), _p(delta), _p(None), _p(weight), _DT[weight.dtype], _p(out), x.shape[0],
                                                 x.shape[1], ctypes.c_float(eps), _DT[out.dtype], self._s()), "add_layernorm")

    def add_layernorm_rows(self, x, delta, rows, weight, eps, out) -> None:
        self.launches += 1
        _check(self._prep_lib().sb_add_layernorm(_p(x), _p(delta), _p(rows), _p(weight), _DT[weight.dtype], _p(out), rows.shape[0],
                                                 x.shape[1], ctypes.c_float(eps), _DT[out.dtype], self._s()), "add_layernorm_rows")

    def add_grouped_rmsnorm(self, x, delta, through, rows, weight, groups: int, eps: float, out) -> None:
        """x += d; out = every one of ``groups`` equal parts of x divided by its own root mean square, times weight (float). d is
        ``delta`` (activations or float), or, with ``through`` (the float weight of such a norm the delta still has to pass), that
        norm of it. With ``rows`` only those rows, and x stays as it is; with x None, out = the norm of delta. ``weight`` None: out =
        x as it is (after the addition)."""
        if (weight is not None and weight.dtype != torch.float32) or (through is not None and through.dtype != torch.float32):
            raise KernelError("add_grouped_rmsnorm: the weights are float")
        self.launches += 1
        n_rows = rows.shape[0] if rows is not None else out.shape[0]
        _check(self._prep_lib().sb_add_grouped_rmsnorm(
            _p(x), _p(delta), _DT[delta.dtype] if delta is not None else 0, _p(through), _p(rows), _p(weight), _p(out), _DT[out.dtype],
            n_rows, out.shape[1], int(groups), ctypes.c_float(eps), self._s()), "grouped norm")

    def poly_norm(self, z, coef, eps: float, out) -> None:
        """out = a N(z) + b N(z^2) + c N(z^3) + e row by row, N dividing a row by its root mean square; coef float [a, b, c, e].
        z and out contiguous and alike; may be the same buffer."""
        if coef.dtype != torch.float32 or z.dtype != out.dtype or z.shape != out.shape or not z.is_contiguous() or not out.is_contiguous():
            raise KernelError("poly_norm: z and out must be contiguous and alike, the coefficients float")
        self.launches += 1
        _check(self._prep_lib().sb_poly_norm(_p(z), _p(coef), ctypes.c_float(eps), _p(out), z.shape[0], z.shape[1], _DT[z.dtype], self._s()),
               "polynomial activation")

    def add_dynamic_tanh(self, x, delta, through, rows, params, out) -> None:
        """x += d; out = tanh(alpha x) w + b with params = float [w | b | alpha]. d is ``delta`` (activations or float), or, with
        ``through`` (the parameters of the dynamic tanh the delta still has to pass), tanh(alpha' delta) w' + b'. With ``rows``
        only those rows, and x stays as it is; with x None, out = the dynamic tanh of delta."""
        self.launches += 1
        n_rows = rows.shape[0] if rows is not None else out.shape[0]
        _check(self._prep_lib().sb_add_dynamic_tanh(_p(x), _p(delta), _DT[delta.dtype] if delta is not None else 0, _p(through), _p(rows),
                                                    _p(params), _p(out), _DT[out.dtype], n_rows, out.shape[1], self._s()), "dynamic tanh")

    _ACTIVATIONS = {"relu_squared": 0, "gelu_tanh": 1, "silu": 2, "tanh": 3}

    def activation(self, x, out, kind: str, bias=None) -> None:
        """out = act(x + bias) element by element, in float, rounded once (x and out contiguous; may be the same buffer)."""
        if not x.is_contiguous() or not out.is_contiguous() or x.shape != out.shape or x.dtype != out.dtype:
            raise KernelError("activation: x and out must be contiguous and alike")
        self.launches += 1
        _check(self._prep_lib().sb_activation(_p(x), _p(bias), _p(out), x.shape[0], x.shape[1], self._ACTIVATIONS[kind], _DT[x.dtype],
                                              self._s()), "activation")

    def linear_activation(self, h, w, out, kind: str) -> None:
        """out = act(h @ w^T), the activation on the product rounded to the activations' type: in bfloat16 in the epilogue of
        the few-rows product or of the tensor-memory product where they take the sizes, else the product and then the
        activation kernel in place."""
        m, n, k = h.shape[0], w.shape[0], h.shape[1]
        if (h.dtype == torch.bfloat16 and out.dtype == torch.bfloat16 and h.stride(0) == k and out.stride(0) == n and w.shape[1] == k
                and tuple(out.shape) == (m, n)):
            code = self._ACTIVATIONS[kind] + 1
            if self.use_skinny_linear and self._core.sb_skinny_linear_supports(m, n, k, 0):
                self.launches += 1
                _check(self._core.sb_skinny_linear_act(_p(h), _p(w), _p(out), m, n, k, code, self._s()), "skinny linear with activation")
                return
            if self._tcgen05_worthwhile(m, n) and self._core.sb_gemm_tcgen05_supports(m, n, k, 0):
                self.launches += 1
                _check(self._core.sb_gemm_tcgen05_act(_p(h), _p(w), _p(out), m, n, k, code, self._wait_flag(), self._s()),
                       "tcgen05 product with activation")
                return
        self.linear(h, w, out)
        self.activation(out, out, kind)

    def add_bias(self, x, bias) -> None:
        """x (float, contiguous) += bias (float) along the rows."""
        if x.dtype != torch.float32 or bias.dtype != torch.float32 or not x.is_contiguous():
            raise KernelError("add_bias: float, contiguous operands")
        self.launches += 1
        _check(self._prep_lib().sb_add_bias(_p(x), _p(bias), x.shape[0], x.shape[1], self._s()), "bias")

    def qk_prepare(self, sums, bias, positions, token_row, heads, kv_heads, head_dim, dim, q_weight, k_weight, eps, inv_freq, rot_dims,
                   q_out, k_cache, v_cache, block_table, page_size, head_norm: bool = False, keys_are_values: bool = False) -> None:
        """From the float sums of a fused query | key | value projection [T, (H + 2 G) * D] (heads padded to D; G = 0: queries only):
        bias added, all queries (all keys) of a token divided by their root mean square over H * dim (G * dim) true elements and
        multiplied by float weights laid out like the padded projection (None: no norm), the first rot_dims elements of every
        query and key head rotated (pairs i, i + rot_dims / 2), queries to q_out, keys and values to their pages. ``head_norm``
        True: instead, every query and key head is divided, after its rotation, by its own root mean square over dim elements;
        "before": before its rotation, and times a weight [D] that all query (all key) heads share. ``keys_are_values``: the row ends
        with the keys, and the value pages take them as projected (bias added)."""
        if sums.dtype != torch.float32:
            raise KernelError("qk_prepare: the projection's sums are float")
        self.launches += 1
        pages = k_cache.shape[0] if k_cache is not None else 0
        _check(self._prep_lib().sb_qk_prepare(
            _p(sums), sums.stride(0), _p(bias), _p(positions), _p(token_row), heads, kv_heads, head_dim, dim, _p(q_weight), _p(k_weight),
            ctypes.c_float(eps), _p(inv_freq), int(rot_dims), _p(q_out), q_out.stride(0), _p(k_cache if kv_heads else None),
            _p(v_cache if kv_heads else None), _p(block_table), block_table.shape[1], page_size, pages, _p(self.errors_tensor()),
            sums.shape[0], _DT[q_out.dtype], 2 if head_norm == "before" else (1 if head_norm else 0), 1 if keys_are_values else 0, self._s()),
            "query/key preparation")

    def linear_batched(self, a, w, out) -> None:
        """out[:, b] = a[:, b] @ w[b]^T for every b: a [M, B, K] and out [M, B, N] may be views of wider buffers (unit stride
        along the last axis), w [B, N, K] is whole. One batched library product."""
        m, b, k = a.shape
        n = w.shape[1]
        if (w.shape[0] != b or w.shape[2] != k or tuple(out.shape) != (m, b, n) or a.dtype != w.dtype or a.stride(2) != 1
                or out.stride(2) != 1 or not w.is_contiguous()):
            raise KernelError(f"linear_batched: a {tuple(a.shape)}, w {tuple(w.shape)}, out {tuple(out.shape)} do not fit")
        self.library_calls += 1
        _check(self._gemm.sb_linear_batched(_p(a), a.stride(0), ctypes.c_longlong(a.stride(1)), _p(w), _p(out), out.stride(0),
                                            ctypes.c_longlong(out.stride(1)), m, n, k, b, _DT[a.dtype], _DT[out.dtype], self._s()),
               "batched linear")

    def gate_up_activation(self, h, w_gate_up, out, activation: str, limit: float = 0.0, alpha: float = 1.0) -> None:
        """out[T, I] = act(h @ w_gate^T, h @ w_up^T), w_gate_up = [w_gate; w_up]: "swiglu", "clamped_swish" (g <- min(g, limit),
        u <- clamp(u, -limit, limit), g * sigmoid(alpha g) * (u + 1)) or "gelu_tanh" (gelu(g) * u, the tanh form); the product is the
        library's or the few-rows kernel's."""
        if activation == "swiglu":
            return self.gate_up_swiglu(h, w_gate_up, out)
        t, inter = h.shape[0], out.shape[1]
        if w_gate_up.shape[0] != 2 * inter or w_gate_up.shape[1] != h.shape[1] or out.shape[0] != t:
            raise KernelError("gate_up_activation: shapes do not fit")
        k = h.shape[1]
        if h.dtype == torch.bfloat16 and out.dtype == torch.bfloat16 and activation == "clamped_swish" and limit > 0.0:
            # the same two fused products as gate_up_swiglu, with the other activation in their epilogues
            if self.use_skinny_linear and self._core.sb_skinny_linear_supports(t, inter, k, 1):
                self.launches += 1
                _check(self._core.sb_skinny_gate_up_clamped(_p(h), _p(w_gate_up), _p(out), t, inter, k, ctypes.c_float(limit),
                                                            ctypes.c_float(alpha), self._s()), "skinny gate/up, clamped")
                return
            if self._tcgen05_worthwhile(t, 2 * inter) and self._core.sb_gemm_tcgen05_supports(t, inter, k, 1):
                self.launches += 1
                _check(self._core.sb_gemm_tcgen05_gate_up_clamped(_p(h), _p(w_gate_up), _p(out), t, inter, k, ctypes.c_float(limit),
                                                                  ctypes.c_float(alpha), self._wait_flag(), self._s()),
                       "tcgen05 gate/up, clamped")
                return
        if h.dtype == torch.bfloat16 and out.dtype == torch.bfloat16 and activation == "gelu_tanh":
            if self.use_skinny_linear and self._core.sb_skinny_linear_supports(t, inter, k, 1):
                self.launches += 1
                _check(self._core.sb_skinny_gate_up_gelu(_p(h), _p(w_gate_up), _p(out), t, inter, k, self._s()), "skinny gate/up, gelu")
                return
            if self._tcgen05_worthwhile(t, 2 * inter) and self._core.sb_gemm_tcgen05_supports(t, inter, k, 1):
                self.launches += 1
                _check(self._core.sb_gemm_tcgen05_gate_up_gelu(_p(h), _p(w_gate_up), _p(out), t, inter, k, self._wait_flag(), self._s()),
                       "tcgen05 gate/up, gelu")
                return
        gate_up = torch.empty((t, 2 * inter), dtype=h.dtype, device=h.device)
        self.linear(h, w_gate_up, gate_up)
        self.launches += 1
        _check(self._prep_lib().sb_gated_activation(_p(gate_up), _p(out), t, inter, {"clamped_swish": 1, "gelu_tanh": 2}[activation], ctypes.c_float(limit),
                                                    ctypes.c_float(alpha), _DT[out.dtype], self._s()), "gated activation")

    def normed_qk_cache_write(self, proj, positions, token_row, heads, kv_heads, head_dim, dim, q_weight, k_weight, eps, temp_coef,
                              temp_every, k_cache, v_cache, block_table, page_size, write_cache) -> None:
        """proj [T, (H + 2 G) * D] (heads padded to D with zeros): queries and keys divided by the root mean square over the
        token's whole projection (H * dim, G * dim true elements) and multiplied by float weights [H * D], [G * D] (None: no
        norm); queries then times 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1), in place; keys and values to the pages."""
        self.launches += 1
        _check(self._prep_lib().sb_normed_qk_cache_write(
            _p(proj), proj.stride(0), _p(positions), _p(token_row), heads, kv_heads, head_dim, dim, _p(q_weight), _p(k_weight),
            ctypes.c_float(eps), ctypes.c_float(temp_coef), int(temp_every), _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1],
            page_size, k_cache.shape[0], 1 if write_cache else 0, _p(self.errors_tensor()), proj.shape[0], _DT[proj.dtype], self._s()),
            "query/key norm and cache write")

    def latent_prepare(self, proj, n_q, positions, token_row, c_weight, eps, inv_freq, rot_dims, heads, dim, rot_dim, rank, head_dim,
                       q_lat, k_cache, block_table, page_size, write_cache, q_off=None, row_out=None,
                       half_pairs: bool = False, latent=None, rot_mult: float = 1.0) -> None:
        """Latent attention between its input product and its attention: proj [T, >= n_q + rank + rot_dim] holds the heads'
        queries ([dim | rot_dim] each), the latent vector and the shared key part. Writes the cache row [normed latent | rotated
        key part | zeros] (if write_cache), the same row into row_out [T, >= rank + rot_dim] (if given), and columns
        [q_off, head_dim) of every head of q_lat (rotated query part, zeros); q_off defaults to rank. Rotated pairs are
        (2 i, 2 i + 1), or with ``half_pairs`` (i, i + rot_dims / 2). ``latent`` [T, >= rank + rot_dim]: the latent vector and the shared
        key part in a buffer of their own (proj then holds the queries only). Cosines and sines are multiplied by ``rot_mult``. With
        neither write_cache nor row_out there is no latent vector: only the queries are prepared (c_weight may be None)."""
        self.launches += 1
        pages = k_cache.shape[0] if k_cache is not None else 0
        _check(self._prep_lib().sb_latent_prepare(
            _p(proj), proj.stride(0), n_q, _p(positions), _p(token_row), _p(c_weight), ctypes.c_float(eps), _p(inv_freq), rot_dims, heads,
            dim, rot_dim, rank, head_dim, _p(q_lat), q_lat.stride(0), rank if q_off is None else q_off, _p(row_out),
            row_out.stride(0) if row_out is not None else 0, _p(k_cache), _p(block_table), block_table.shape[1], page_size, pages,
            1 if write_cache else 0, _p(self.errors_tensor()), proj.shape[0], _DT[proj.dtype], 1 if half_pairs else 0, _p(latent),
            latent.stride(0) if latent is not None else 0, ctypes.c_float(rot_mult), self._s()),
            "latent attention preparation")

    def linear(self, a, w, out) -> None:
        """out[M,N] = a[M,K] @ w[N,K]^T (library matrix product)."""
        if a.dtype != w.dtype or a.shape[1] != w.shape[1] or out.shape[0] != a.shape[0] or out.shape[1] != w.shape[0]:
            raise KernelError(f"linear: a {tuple(a.shape)} {a.dtype}, w {tuple(w.shape)} {w.dtype}, out {tuple(out.shape)} do not fit")
        m, n, k = a.shape[0], w.shape[0], a.shape[1]
        if a.stride(0) != k or out.stride(0) != n:
            # a column slice of a wider buffer on either side: the library takes the row strides
            if a.stride(1) != 1 or out.stride(1) != 1:
                raise KernelError("linear: operands must be contiguous along their rows")
            self.library_calls += 1
            _check(self._gemm.sb_linear_ld(_p(a), a.stride(0), _p(w), _p(out), out.stride(0), m, n, k, _DT[a.dtype], _DT[out.dtype],
                                           self._s()), "linear")
            return
        key = (a.dtype, out.dtype, m, n, k, self.use_skinny_linear, self.use_tcgen05, self.TCGEN05_MIN_TILES, self.tcgen05_for_plain_products, 0)
        route = self._routes.get(key)
        if route is None:
            route = 0
            if a.dtype == torch.bfloat16 and self.use_skinny_linear and self._core.sb_skinny_linear_supports(m, n, k, 0):
                route = 1
            elif (a.dtype == torch.bfloat16 and out.dtype == torch.bfloat16 and self.tcgen05_for_plain_products
                    and self._tcgen05_worthwhile(m, n) and self._core.sb_gemm_tcgen05_supports(m, n, k, 0)):
                route = 2
            elif (a.dtype == torch.float32 and out.dtype == torch.float32 and self.use_skinny_linear
                    and self._core.sb_skinny_linear_f32_supports(m, n, k)):
                route = 3
            self._routes[key] = route
        if route == 1:
            self.launches += 1
            _check(self._core.sb_skinny_linear(_p(a), _p(w), _p(out), m, n, k, _DT[out.dtype], 0, self._s()), "skinny linear")
        elif route == 2:
            self.launches += 1
            _check(self._core.sb_gemm_tcgen05(_p(a), _p(w), _p(out), m, n, k, 0, self._wait_flag(), self._s()), "tcgen05 product")
        elif route == 3:
            self.launches += 1
            _check(self._core.sb_skinny_linear_f32(_p(a), _p(w), _p(out), m, n, k, self._s()), "skinny linear, float32")
        else:
            self.library_calls += 1
            _check(self._gemm.sb_linear(_p(a), _p(w), _p(out), m, n, k, _DT[a.dtype], _DT[out.dtype], self._s()), "linear")

    def gate_up_swiglu(self, h, w_gate_up, out) -> None:
        """out[T, I] = silu(h @ w_gate^T) * (h @ w_up^T), w_gate_up = [w_gate; w_up] of shape [2I, K]."""
        t, inter, k = h.shape[0], out.shape[1], h.shape[1]
        if w_gate_up.shape[0] != 2 * inter or w_gate_up.shape[1] != k or out.shape[0] != t:
            raise KernelError("gate_up_swiglu: shapes do not fit")
        key = (h.dtype, out.dtype, t, inter, k, self.use_skinny_linear, self.use_tcgen05, self.TCGEN05_MIN_TILES, 1)
        route = self._routes.get(key)
        if route is None:
            route = 0
            if h.dtype == torch.bfloat16 and self.use_skinny_linear and self._core.sb_skinny_linear_supports(t, inter, k, 1):
                route = 1
            elif (h.dtype == torch.bfloat16 and self._tcgen05_worthwhile(t, 2 * inter)
                    and self._core.sb_gemm_tcgen05_supports(t, inter, k, 1)):
                route = 2
            self._routes[key] = route
        if route == 1:
            self.launches += 1
            _check(self._core.sb_skinny_linear(_p(h), _p(w_gate_up), _p(out), t, inter, k, _DT[out.dtype], 1, self._s()),
                   "skinny gate/up")
            return
        if route == 2:
            self.launches += 1
            _check(self._core.sb_gemm_tcgen05(_p(h), _p(w_gate_up), _p(out), t, inter, k, 1, self._wait_flag(), self._s()),
                   "tcgen05 gate/up")
            return
        gate_up = torch.empty((t, 2 * inter), dtype=h.dtype, device=h.device)
        self.linear(h, w_gate_up, gate_up)
        self.swiglu(gate_up, out)

    def swiglu(self, gate_up, out) -> None:
        self.launches += 1
        _check(self._core.sb_swiglu(_p(gate_up), _p(out), out.shape[0], out.shape[1], _DT[out.dtype], self._s()), "swiglu")

    def rope_cache_write(self, qkv, positions, token_row, inv_freq, pairing, rotary_dim, heads, kv_heads, head_dim,
                         k_cache, v_cache, block_table, page_size, write_cache) -> None:
        self.launches += 1
        num_pages = k_cache.shape[0] if k_cache is not None else 0
        _check(self._core.sb_rope_cache_write(
            _p(qkv), _p(positions), _p(token_row), _p(inv_freq), pairing, rotary_dim, heads, kv_heads, head_dim,
            _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], page_size, num_pages,
            1 if write_cache else 0, _p(self.errors_tensor()), qkv.shape[0], _DT[qkv.dtype], self._s()), "rope_cache_write")

    def qkv_rope_cache(self, h, w_qkv, qkv, positions, token_row, inv_freq, pairing, rotary_dim, heads, kv_heads, head_dim,
                       k_cache, v_cache, block_table, page_size, write_cache, memo=None) -> None:
        """qkv = h @ w_qkv^T, queries and keys rotated, keys and values written to the cache pages.

        In bfloat16 with adjacent rotary pairs this is one kernel, for a handful of rows and for many (the product with
        rotation and cache write in its epilogue; only the query columns of ``qkv`` are then written). Otherwise, and
        for row counts in between that go to the library, the product and the rotary kernel run one after the other.
        ``memo``: a dict that lives as long as the step's positions do; what depends on them alone is kept there."""
        m, k = h.shape
        n = qkv.shape[1]
        if (h.dtype == torch.bfloat16 and self.use_skinny_linear and self.fuse_rope and pairing == 1 and head_dim % 8 == 0
                and self._core.sb_skinny_linear_supports(m, n, k, 0)):
            self.launches += 1
            _check(self._core.sb_skinny_qkv_rope(
                _p(h), _p(w_qkv), _p(qkv), m, k, _p(positions), _p(token_row), _p(inv_freq), rotary_dim, heads, kv_heads, head_dim,
                _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], page_size, k_cache.shape[0],
                1 if write_cache else 0, _p(self.errors_tensor()), self._s()), "q/k/v product with rotation")
            return
        if (h.dtype == torch.bfloat16 and qkv.dtype == torch.bfloat16 and self.fuse_rope and pairing == 1
                and self._tcgen05_worthwhile(m, n)
                and self._core.sb_gemm_tcgen05_qkv_rope_supports(m, k, rotary_dim, heads, kv_heads, head_dim)):
            # many rows: the tensor-memory product with the same epilogue; cosines and sines from a table that the
            # first layer of the step makes and the others find in the step's memo
            key = ("rope_angles", inv_freq.data_ptr(), positions.data_ptr(), rotary_dim)
            angles = memo.get(key) if memo is not None else None
            if angles is None:
                angles = torch.empty((max(rotary_dim // 2, 1), m, 2), dtype=torch.float32, device=h.device)
                self.launches += 1
                _check(self._core.sb_rope_angles(_p(positions), _p(inv_freq), rotary_dim, m, _p(angles), self._s()), "rotary angles")
                if memo is not None:
                    memo[key] = angles
            self.launches += 1
            _check(self._core.sb_gemm_tcgen05_qkv_rope(
                _p(h), _p(w_qkv), _p(qkv), m, k, _p(positions), _p(token_row), _p(angles), rotary_dim, heads, kv_heads, head_dim,
                _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], page_size, k_cache.shape[0],
                1 if write_cache else 0, _p(self.errors_tensor()), self._wait_flag(), self._s()),
                "tcgen05 q/k/v product with rotation")
            return
        self.linear(h, w_qkv, qkv)
        self.rope_cache_write(qkv, positions, token_row, inv_freq, pairing, rotary_dim, heads, kv_heads, head_dim,
                              k_cache, v_cache, block_table, page_size, write_cache)

    def attention(self, qkv, k_cache, v_cache, block_table, cu_q, kv_len, token_row, positions, heads, kv_heads, head_dim,
                  page_size, scale, window, out, shape, slopes=None, chunk: int = 0, softcap: float = 0.0, sinks=None,
                  keep_first: int = 0) -> None:
        """``slopes`` (float [heads]): slope_h * distance is taken off every score; ``chunk`` > 0: a query sees only the keys of
        its own block of ``chunk`` positions; ``softcap`` c > 0: a scaled score s becomes c * tanh(s / c); ``sinks`` (float
        [heads]): exp(sink_h) joins the softmax's denominator; ``keep_first`` n > 0 (with a window): the sequence's first n keys
        stay visible to every later query. In bfloat16 all run on the mma.sync kernels; cap and sink
        also on the tensor-memory kernel (prompt portions at head sizes 64 and 128); in float32 on the plain-arithmetic kernel."""
        lib = self._attention_lib(head_dim)
        softcap = float(softcap or 0.0)
        keep_first = int(keep_first or 0) if window else 0
        opts = slopes is not None or chunk or softcap > 0.0 or sinks is not None or keep_first > 0
        if opts and qkv.dtype == torch.bfloat16 and not self.force_simt_attention:
            return self._attention_mma(lib, qkv, k_cache, v_cache, block_table, cu_q, kv_len, heads, kv_heads, head_dim,
                                       page_size, scale, window, out, shape, slopes=slopes, chunk=int(chunk), softcap=softcap, sinks=sinks,
                                       keep_first=keep_first)
        if opts:
            group = heads // kv_heads
            self.launches += (1 if group <= 16 else 0) + (1 if group > 16 or shape.max_q * group > 16 else 0)
            _check(lib.sb_attention_simt_keep(
                _p(qkv), qkv.stride(0), _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], _p(cu_q), _p(kv_len),
                heads, kv_heads, page_size, k_cache.shape[0], ctypes.c_float(scale), window, _p(out), shape.rows, shape.max_q,
                _DT[qkv.dtype], _p(slopes), int(chunk), ctypes.c_float(softcap), _p(sinks), keep_first, self._s()),
                "attention with score options")
            return
        if qkv.dtype == torch.bfloat16 and not self.force_simt_attention:
            return self._attention_mma(lib, qkv, k_cache, v_cache, block_table, cu_q, kv_len, heads, kv_heads, head_dim,
                                       page_size, scale, window, out, shape)
        group = heads // kv_heads
        # requests of at most 16 rows run in the decoding shape, the others in tiles: one launch each, as needed
        self.launches += (1 if group <= 16 else 0) + (1 if group > 16 or shape.max_q * group > 16 else 0)
        _check(lib.sb_attention_simt(
            _p(qkv), qkv.shape[1], _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], _p(cu_q), _p(kv_len),
            heads, kv_heads, page_size, k_cache.shape[0], ctypes.c_float(scale), window, _p(out), shape.rows, shape.max_q,
            _DT[qkv.dtype], self._s()), "attention")

    # Thread blocks of the deep shape that the key splits of a batch should fill: one per SM (set from the device's
    # SM count when the kernels are loaded; 148 on a B200).
    TARGET_BLOCKS = 148
    MAX_SPLITS = 32
    # query heads per group when all heads share one cached row per token (SERVE_B200_LATENT_GROUP for measurements)
    LATENT_GROUP = int(os.environ.get("SERVE_B200_LATENT_GROUP", "8"))
    LATENT_GROUP_DECODE = int(os.environ.get("SERVE_B200_LATENT_GROUP_DECODE", "4"))

    def split_plan(self, rows: int, kv_heads: int, max_kv: int) -> int:
        """Number of key splits of the deep shape for a batch; a function of sizes only, never of data.
        (Each request's own length is then shared out evenly over the splits inside the kernel.)"""
        want = max(1, self.TARGET_BLOCKS // max(1, rows * kv_heads))
        return max(1, min(want, -(-max_kv // 256), self.MAX_SPLITS))

    def _attention_mma(self, lib, qkv, k_cache, v_cache, block_table, cu_q, kv_len, heads, kv_heads, head_dim, page_size,
                       scale, window, out, shape, slopes=None, chunk: int = 0, softcap: float = 0.0, sinks=None,
                       keep_first: int = 0) -> None:
        # One cached row for many query heads (keys and values the same tensor): the heads are dealt to groups of LATENT_GROUP
        # that each count as a kv head reading the same rows. A decoding request is then several (request, kv head) pairs of
        # few rows, which the deep shape spreads over the SMs with its key splits; as one pair of 32 rows it would be a single
        # block of the wide shape walking all keys alone. For prompt portions the grouping changes neither work nor traffic.
        kv_div = 1
        if k_cache is v_cache:
            # (a step of single tokens takes smaller groups: measured at batch 8 after 2,048 tokens, groups of 4 against 8 give
            # 29 against 38 us a launch with 8 heads and 31 against 39 us with 16)
            per_group = self.LATENT_GROUP_DECODE if shape.max_q == 1 else self.LATENT_GROUP
            if kv_heads * per_group < heads and heads % (kv_heads * per_group) == 0:
                kv_div = heads // (kv_heads * per_group)
                kv_heads = kv_heads * kv_div
        group = heads // kv_heads
        min_q = getattr(shape, "min_q", 1)
        which = 0
        if group > 16 or shape.max_q * group > 16:
            which |= 1
        if group <= 16 and min_q * group <= 16:
            which |= 2
            if group > 8 or (shape.max_q > 1 and min(shape.max_q, 16 // group) * group > 8):
                which |= 4      # some request of the deep shape may have more than 8 rows
                neg_q = getattr(shape, "neg_q_sorted", None)
                if neg_q is not None and group <= 8:
                    # the step says how many tokens each request brings: is any count in (8 // group, 16 // group]?
                    if bisect.bisect_left(neg_q, -(8 // group)) == bisect.bisect_left(neg_q, -(16 // group)):
                        which &= ~4
        # requests of the wide shape (more than 16 // group tokens): only they get blocks, if the step says who they are
        wide_rows, n_wide = None, 0
        neg_q = getattr(shape, "neg_q_sorted", None)
        if (which & 1) and neg_q is not None and getattr(shape, "rows_by_q", None) is not None:
            n_wide = bisect.bisect_left(neg_q, -(16 // group) if group <= 16 else 0)
            wide_rows = shape.rows_by_q
        num_splits, scratch, tickets = 1, None, None
        if which & 2:
            # (behind a window a query reads at most the window's keys and the kept first ones, however long the sequence)
            num_splits = self.split_plan(shape.rows, kv_heads, min(shape.max_kv, window + keep_first + 16) if window else shape.max_kv)
            if num_splits > 1:
                scratch = self._scratch_buffer(lib, shape.rows, kv_heads, num_splits)
                tickets = self._ticket_buffer(shape.rows * kv_heads)
        by_distance = slopes is not None or chunk > 0 or softcap > 0.0 or sinks is not None
        if (which & 1) and slopes is None and not chunk and not keep_first and kv_div == 1 and self.use_tcgen05_attention and self._tc_attention_takes(lib, heads, kv_heads, head_dim, page_size, window, qkv.shape[1]):
            # prompt portions on the tensor-memory path; what is left (decoding rows) goes to the deep shape below
            self.launches += 1
            _check(lib.sb_attention_tc_opts(
                _p(qkv), qkv.shape[1], qkv.shape[0], _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], _p(cu_q),
                _p(kv_len), heads, kv_heads, page_size, k_cache.shape[0], ctypes.c_float(scale), _p(out),
                n_wide if wide_rows is not None else shape.rows, shape.max_q, _p(wide_rows), self._wait_flag(),
                ctypes.c_float(softcap), _p(sinks), self._s()), "tcgen05 attention")
            which &= ~1
            if not which:
                return
        self.launches += (which & 1) + ((which >> 1) & 1) + ((which >> 2) & 1)
        _check(lib.sb_attention_mma_keep(
            _p(qkv), qkv.stride(0), _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], _p(cu_q), _p(kv_len),
            heads, kv_heads, page_size, k_cache.shape[0], ctypes.c_float(scale), window, _p(out), shape.rows, shape.max_q,
            which, int(shape.max_kv), num_splits, _p(scratch), _p(tickets), _p(wide_rows), n_wide, _p(slopes), chunk,
            ctypes.c_float(softcap), _p(sinks), kv_div, keep_first, self._s()), "attention")

    # Scratch bytes a launch of the mixed-head attention may use; a step that needs more runs in runs of tokens.
    TALK_SCRATCH_BYTES = int(os.environ.get("SERVE_B200_TALK_SCRATCH", str(1 << 30)))

    def talking_attention(self, q, k_cache, v_cache, block_table, cu_q, kv_len, positions, heads, kv_heads, head_dim, page_size, scale,
                          talk, out, shape, chunk: int = 0, softcap: float = 0.0, sinks=None) -> None:
        """Attention whose heads' softmax weights are mixed before they meet the values: weight_h = sum_g talk[h, g] weight_g, head h
        then reads the values of its own kv head. q [T, H * D]; ``talk`` of q's type: [H, H] in float32, in bfloat16 [Hp, Hp] with Hp
        the next multiple of 16 and zeros beyond H. chunk, softcap and sinks as in ``attention``."""
        lib = self._talk_lib(head_dim)
        group = heads // kv_heads
        t = q.shape[0]
        bf16 = q.dtype == torch.bfloat16
        if talk.dtype != q.dtype or talk.shape[0] != (16 * -(-heads // 16) if bf16 else heads) or not talk.is_contiguous():
            raise KernelError("talking_attention: the mixing matrix has the queries' type, padded to a multiple of 16 in bfloat16")
        # the most keys a token can read, counted from the tile of 64 its first key lies in
        max_keys = min(chunk + 63, shape.max_kv) if chunk else shape.max_kv
        pitch = 64 * -(-max_keys // 64)
        which = 0
        if group > 16 or shape.max_q * group > 16:
            which |= 1
        if group <= 16 and getattr(shape, "min_q", 1) * group <= 16:
            which |= 2
        wide_rows, n_wide = None, 0
        neg_q = getattr(shape, "neg_q_sorted", None)
        if (which & 1) and neg_q is not None and getattr(shape, "rows_by_q", None) is not None:
            n_wide = bisect.bisect_left(neg_q, -(16 // group) if group <= 16 else 0)
            wide_rows = shape.rows_by_q
        per_token = heads * (pitch * (4 + q.element_size()) + pitch // 64 * 8)
        step = max(1, min(t, self.TALK_SCRATCH_BYTES // per_token))
        n_splits, part, tickets = 1, None, None
        if bf16 and which & 2:
            n_splits = max(1, min(-(-4 * self.TARGET_BLOCKS // (shape.rows * kv_heads)), -(-pitch // 128), self.MAX_SPLITS))
            if n_splits > 1:
                part = torch.empty((shape.rows, kv_heads, n_splits, 16, head_dim), dtype=torch.float32, device=q.device)
                tickets = self._ticket_buffer(shape.rows * kv_heads)
        e = torch.empty((step, heads, pitch), dtype=torch.float32, device=q.device)
        stats = torch.empty((step, heads, pitch // 64, 2), dtype=torch.float32, device=q.device)
        w = torch.empty((step, heads, pitch), dtype=q.dtype, device=q.device)
        for t0 in range(0, t, step):
            separate_mix = which & 1 or shape.rows * kv_heads > self.TARGET_BLOCKS      # (else the values' kernel mixes)
            self.launches += 2 * ((which & 1) + ((which >> 1) & 1)) + (1 if separate_mix else 0) if bf16 else 3
            _check(lib.sb_talking_attention(
                _p(q), q.stride(0), _p(k_cache), _p(v_cache), _p(block_table), block_table.shape[1], _p(cu_q), _p(kv_len), _p(positions),
                heads, kv_heads, page_size, k_cache.shape[0], ctypes.c_float(scale), ctypes.c_float(float(softcap or 0.0)), int(chunk or 0),
                _p(sinks), _p(talk), _p(e), _p(stats), _p(w), pitch, t0, min(t0 + step, t), _p(out), shape.rows, shape.max_q, max_keys, which,
                _p(wide_rows), n_wide, n_splits, _p(part), _p(tickets), t, self._wait_flag(), 1 if self.use_tcgen05_attention else 0, _DT[q.dtype],
                self._s()), "attention with mixed heads")

    def _tc_attention_takes(self, lib, heads, kv_heads, head_dim, page_size, window, stride) -> bool:
        key = (heads, kv_heads, head_dim, page_size, window, stride)
        ok = self._tc_attention_ok.get(key)
        if ok is None:
            ok = self._tc_attention_ok[key] = bool(lib.sb_attention_tc_supports(heads, kv_heads, page_size, window, stride))
        return ok

    def _scratch_buffer(self, lib, rows: int, kv_heads: int, num_splits: int) -> torch.Tensor:
        """Float scratch for the partial results of split keys. Launches on one stream follow one another, so one buffer
        serves all layers and steps; a larger one is made when needed and the old one stays alive for captured graphs."""
        need = lib.sb_attention_mma_scratch_bytes(rows, kv_heads, num_splits) // 4
        if self._split_scratch is None or self._split_scratch.numel() < need:
            if self._split_scratch is not None:
                self._keep.append(self._split_scratch)
            self._split_scratch = torch.empty(max(need, 1 << 20), dtype=torch.float32, device=self.device)
        return self._split_scratch

    def _ticket_buffer(self, n: int) -> torch.Tensor:
        """A zeroed int32 buffer of at least n entries. Every launch leaves it zeroed, so one buffer serves all
        layers and steps; a larger one is made when needed and the old ones stay alive for captured graphs."""
        if not self._tickets or self._tickets[-1].numel() < n:
            self._tickets.append(torch.zeros(max(n, 4096), dtype=torch.int32, device=self.device))
        return self._tickets[-1]

    # ---- whole layers of a decoding step in one launch ---------------------------------------------------------------
    def _stack_lib(self, head_dim: int):
        lib = self._stack.get(head_dim)
        if lib is None:
            job = layer_run_job(head_dim)
            job["verbose"] = self._verbose
            path = build.build_library(**job)
            self.paths[job["name"]] = path
            lib = self._stack[head_dim] = ctypes.CDLL(path)
            lib.sb_decode_stack_partial_floats.restype = ctypes.c_longlong
            if lib.sb_decode_stack_layer_bytes() != _STACK_LAYER.itemsize:
                raise KernelError("the layer table's layout on the host and in the library differ")
        return lib

    def plan_layer_run(self, descs):
        """(n, plan): the first n of the described layers can run as one launch in a decoding step (n may be 0).
        ``descs``: what Block.fused_description gives, one per layer in running order."""
        first = descs[0]
        if not self._layer_run_describable(first):
            return 0, None
        att, ff = first["mixer"], first["feed_forward"]
        key = (att["hidden"], att["heads"], att["kv_heads"], att["head_dim"], ff["intermediate"], att["page_size"])
        n = 0
        groups = []
        for d in descs:
            if not self._layer_run_describable(d):
                break
            a, f = d["mixer"], d["feed_forward"]
            if (a["hidden"], a["heads"], a["kv_heads"], a["head_dim"], f["intermediate"], a["page_size"]) != key:
                break
            if a["group"] not in groups:
                if len(groups) == _STACK_MAX_GROUPS:
                    break
                groups.append(a["group"])
            n += 1
        if n == 0:
            return 0, None
        hidden, heads, kv_heads, head_dim, inter, page_size = key
        lib = self._stack_lib(head_dim)
        blocks = lib.sb_decode_stack_blocks()
        if blocks <= 0 or not lib.sb_decode_stack_supports(1, hidden, heads, kv_heads, inter, blocks):
            return 0, None
        table = np.zeros(n, dtype=_STACK_LAYER)
        keep = []
        for i, d in enumerate(descs[:n]):
            a, f, n1, n2 = d["mixer"], d["feed_forward"], d["mixer_norm"], d["feed_forward_norm"]
            row = table[i]
            row["wqkv"], row["wo"] = a["w_qkv"].data_ptr(), a["w_o"].data_ptr()
            row["wgu"], row["wdown"] = f["w_gate_up"].data_ptr(), f["w_down"].data_ptr()
            row["norm1"], row["norm2"] = n1["weight"].data_ptr(), n2["weight"].data_ptr()
            row["inv_freq"] = a["inv_freq"].data_ptr()
            row["kc"], row["vc"] = a["k"].data_ptr(), a["v"].data_ptr()
            row["eps1"], row["eps2"] = n1["eps"], n2["eps"]
            row["scale_log2"] = a["scale"] * 1.4426950408889634
            row["rot"], row["window"] = a["rotary_dim"], a["window"]
            row["norm_f32"] = (1 if n1["weight"].dtype == torch.float32 else 0) | (2 if n2["weight"].dtype == torch.float32 else 0)
            row["group"] = groups.index(a["group"])
            row["num_pages"] = a["k"].shape[0]
            row["write_cache"] = 1 if a["writes"] else 0
            keep.extend([a["w_qkv"], a["w_o"], f["w_gate_up"], f["w_down"], n1["weight"], n2["weight"], a["inv_freq"], a["k"], a["v"]])
        dev_table = torch.from_numpy(table.view(np.uint8).copy()).to(self.device)
        return n, LayerRunPlan(lib, dev_table, keep, n, hidden, heads, kv_heads, head_dim, inter, groups, page_size, blocks)

    @staticmethod
    def _layer_run_describable(d) -> bool:
        if d is None or d.get("kind") != "pre_norm":
            return False
        a, f, n1, n2 = d.get("mixer"), d.get("feed_forward"), d.get("mixer_norm"), d.get("feed_forward_norm")
        if not (a and f and n1 and n2) or a.get("kind") != "attention" or f.get("kind") != "swiglu":
            return False
        if n1.get("kind") != "rms" or n2.get("kind") != "rms":
            return False
        if a["head_dim"] not in LAYER_RUN_HEAD_DIMS or a["w_qkv"].dtype != torch.bfloat16 or a["k"] is None or a["k"].dtype != torch.bfloat16:
            return False
        if a["rotary_dim"] > 0 and a["pairing"] != 1:
            return False
        if a["rotary_dim"] % 2 or n1["size"] != a["hidden"] or n2["size"] != a["hidden"] or f["hidden"] != a["hidden"]:
            return False
        return all(n["weight"].dtype in (torch.float32, torch.bfloat16) for n in (n1, n2))

    def layer_run_takes(self, plan: LayerRunPlan, ctx) -> bool:
        """Does this step go through the one-launch kernel? Decoding steps (one token per request) of at most 16 requests."""
        shape = ctx.shape
        if not (self.use_layer_runs and shape.pure_decode and shape.tokens <= _STACK_MAX_ROWS):
            return False
        ok = plan.takes.get(shape.tokens)
        if ok is None:
            ok = plan.takes[shape.tokens] = bool(plan.lib.sb_decode_stack_supports(shape.tokens, plan.hidden, plan.heads, plan.kv_heads,
                                                                                  plan.inter, plan.blocks))
        return ok

    def layer_run(self, plan: LayerRunPlan, x, pending, ctx):
        """Runs the plan's layers on the step's tokens: x [M, hidden] float32 is updated in place; returns (x, pending)."""
        m = x.shape[0]
        dev = x.device
        act = lambda cols: torch.empty((m, cols), dtype=torch.bfloat16, device=dev)
        n_qkv = (plan.heads + 2 * plan.kv_heads) * plan.head_dim
        x_scratch = torch.empty_like(x)
        delta_o, delta_down = act(plan.hidden), act(plan.hidden)
        qkv, attn, inter = act(n_qkv), act(plan.heads * plan.head_dim), act(plan.inter)
        num_splits = max(1, min(plan.blocks // max(1, m * plan.kv_heads), -(-ctx.shape.max_kv // 256), self.MAX_SPLITS))
        partials = tickets = None
        if num_splits > 1:
            need = plan.lib.sb_decode_stack_partial_floats(_STACK_MAX_ROWS, plan.kv_heads, self.MAX_SPLITS)
            if self._stack_partials is None or self._stack_partials.numel() < need:
                self._stack_partials = torch.empty(need, dtype=torch.float32, device=self.device)
                self._keep.append(self._stack_partials)
            partials = self._stack_partials
            tickets = self._ticket_buffer(m * plan.kv_heads)
        if self._stack_sync is None:
            self._stack_sync = torch.zeros(4, dtype=torch.int32, device=self.device)
        tables = (ctypes.c_void_p * _STACK_MAX_GROUPS)()
        widths = (ctypes.c_int * _STACK_MAX_GROUPS)()
        for i, g in enumerate(plan.groups):
            tables[i] = ctx.block_tables[g].data_ptr()
            widths[i] = ctx.block_tables[g].shape[1]
        self.launches += 1
        self.layer_runs += 1
        _check(plan.lib.sb_decode_stack(
            _p(plan.table), plan.n_layers, m, plan.hidden, plan.heads, plan.kv_heads, plan.inter, _p(ctx.positions), _p(ctx.kv_len),
            tables, widths, len(plan.groups), plan.page_size, _p(x), _p(x_scratch), _p(pending), _p(delta_o), _p(delta_down),
            _p(qkv), _p(attn), _p(inter), _p(partials), _p(tickets), num_splits, _p(self._stack_sync), _p(self.errors_tensor()),
            plan.blocks, _p(self.layer_run_timing), self._s()), "layers of a decoding step")
        return x, delta_down

    # ---- mixers with recurrent state, routed experts ------------------------------------------------------------------
    def _seq_lib(self):
        if self._seq is None:
            job = sequence_job()
            job["verbose"] = self._verbose
            path = build.build_library(**job)
            self.paths[job["name"]] = path
            self._seq = ctypes.CDLL(path)
        return self._seq

    def _moe_lib(self):
        if self._moe is None:
            job = experts_job()
            job["verbose"] = self._verbose
            path = build.build_library(**job)
            self.paths[job["name"]] = path
            self._moe = ctypes.CDLL(path)
        return self._moe

    def _prep_lib(self):
        if self._prep is None:
            job = projection_job()
            job["verbose"] = self._verbose
            path = build.build_library(**job)
            self.paths[job["name"]] = path
            self._prep = ctypes.CDLL(path)
        return self._prep

    def causal_conv(self, x, weight, bias, state, ctx, out, activation: str = "none", residual: bool = False) -> None:
        """out[t] = act(bias + sum_j weight[:, j] * x[t - taps + 1 + j] (+ x[t])) per channel, over each request's own tokens;
        the taps - 1 inputs before a portion come from ``state`` [slots, taps - 1, C] (float), which then takes the portion's
        last ones. x and out may be column slices (row strides are passed on)."""
        c, taps = weight.shape
        self.launches += 1 if (ctx.shape.pure_decode or taps == 1) else 2
        _check(self._seq_lib().sb_causal_conv(
            _p(x), x.stride(0), _p(weight), _p(bias), _p(state), _p(ctx.slots), _p(ctx.cu_q), _p(ctx.token_row), _p(out), out.stride(0),
            c, taps, {"none": 0, "silu": 1}[activation], 1 if residual else 0, x.shape[0], ctx.shape.rows,
            1 if ctx.shape.pure_decode else 0, ctypes.c_longlong(state.stride(0) if state is not None else 0), _DT[x.dtype], self._s()),
            "short convolution")

    def token_shift_mix(self, x, mu, state, ctx, out) -> None:
        """out[m, t] = x[t] + (x[t - 1] - x[t]) * mu[m] over each request's own tokens; before a portion's first token stands
        ``state`` [slots, 1, C] (float), which then takes the portion's last input. out [n_mix, T, C]."""
        c = x.shape[1]
        if mu.dtype != torch.float32 or mu.shape[1] != c or tuple(out.shape) != (mu.shape[0], x.shape[0], c) or out.stride(2) != 1 or x.stride(1) != 1:
            raise KernelError("token_shift_mix: shapes do not fit")
        self.launches += 1 if ctx.shape.pure_decode else 2
        _check(self._seq_lib().sb_token_shift(
            _p(x), x.stride(0), _p(mu), mu.shape[0], _p(state), ctypes.c_longlong(state.stride(0)), _p(ctx.slots), _p(ctx.cu_q),
            _p(ctx.token_row), _p(out), ctypes.c_longlong(out.stride(0)), out.stride(1), c, x.shape[0], ctx.shape.rows,
            1 if ctx.shape.pure_decode else 0, _DT[x.dtype], self._s()), "token shift")

    def linear_recurrence(self, mode: str, q, k, v, state, ctx, out, heads: int, qk_heads: int, dk: int, dv: int, aux=None, rate=None,
                          decay=None, a_log=None, dt_bias=None, d_skip=None, q_scale: float = 1.0, rate_per_head: bool = False,
                          bonus=None, rate_scale: float = 1.0, inv_freq=None, rot_dims: int = 0, k_scale: float = 1.0) -> None:
        """One matrix state [dk, dv] per (request, head), walked over the step's tokens: see csrc/sequence_ops.cu.
        mode "decay": S = decay_h S + k v^T with silu on q, k, v; "ssm": S = exp(-exp(a_log) dt) S + dt k v^T, dt =
        softplus(aux + dt_bias), o += d_skip v; "delta": S = g S, S += k (beta (v - S^T k))^T with g = exp(-exp(a_log)
        softplus(rate + dt_bias)), beta = sigmoid(aux), q and k made unit vectors (``rate_per_head``: rate [T, heads] and dt_bias
        [heads], one decay for a head's whole state); "wkv": o = S^T q + (sum_i q_i bonus_i k_i) v, then S = diag(d) S + k v^T
        with d = exp(-exp(rate + dt_bias)) per row (rate [T, heads * dk], of a dtype of its own; bonus float [heads * dk]);
        "gla": S = diag(a) S + k v^T, o = S^T (q_scale q), a = sigmoid(rate + dt_bias)^rate_scale per row (rate [T, heads * dk]);
        "retention": S = decay_h S + k v^T on q, k, v as they are, the first rot_dims elements of q and k rotated by the tokens'
        positions (pairs i, i + rot_dims / 2; inv_freq float [rot_dims / 2]), k times k_scale.
        out: float [T, heads * dv]. In bfloat16, requests that bring more than CHUNKED_FROM tokens run "retention" chunk by chunk on
        the tensor cores (csrc/chunked_retention.cu), the others token by token."""
        max_walk = 0
        if mode == "retention" and self._chunked_retention(q, k, v, state, ctx, out, heads, dk, dv, decay, inv_freq, rot_dims, k_scale):
            if getattr(ctx.shape, "min_q", 1) > self.CHUNKED_FROM:
                return
            max_walk = self.CHUNKED_FROM
        par = a_log if a_log is not None else (dt_bias if mode == "gla" else None)
        lib = self._seq_lib()
        code = {"decay": 0, "ssm": 1, "delta": 2, "wkv": 3, "gla": 4, "retention": 5}[mode]
        lib.sb_linear_recurrence_work_floats.restype = ctypes.c_longlong
        need = lib.sb_linear_recurrence_work_floats(code, q.shape[0], heads, qk_heads, dk, dv)
        if need < 0:
            raise KernelError(f"linear recurrence: a state of {dk} rows is beyond the kernel's 512")
        work = torch.empty(need, dtype=torch.float32, device=q.device)       # what the first kernel leaves for the second
        self.launches += 2
        _check(lib.sb_linear_recurrence(
            code, _p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0),
            _p(aux), aux.stride(0) if aux is not None else 0, _p(rate), rate.stride(0) if rate is not None else 0,
            _DT[rate.dtype] if rate is not None else 0, 1 if rate_per_head else 0, _p(bonus), _p(decay),
            _p(a_log), _p(dt_bias), _p(d_skip), _DT[par.dtype] if par is not None else 0, _p(state), _p(ctx.slots), _p(ctx.cu_q),
            _p(out), out.stride(0), heads, qk_heads, dk, dv, ctypes.c_float(q_scale), ctx.shape.rows, q.shape[0], _p(work),
            ctypes.c_longlong(state.stride(0)), _DT[v.dtype], ctypes.c_float(rate_scale), _p(ctx.positions), _p(inv_freq), int(rot_dims),
            ctypes.c_float(k_scale), _p(ctx.token_row), max_walk, self._s()), "linear recurrence")

    # Requests with more tokens than this go through the chunked kernels, where those take the layout.
    CHUNKED_FROM = 32
    use_chunked_retention = True             # tests: False keeps every request on the walking kernel

    def _chunked_retention(self, q, k, v, state, ctx, out, heads, dk, dv, decay, inv_freq, rot_dims, k_scale) -> bool:
        """Run the recurrence of the step's longer requests chunk by chunk, if there are any and the kernels take the layout."""
        shape = ctx.shape
        if not self.use_chunked_retention or q.dtype != torch.bfloat16 or shape.max_q <= self.CHUNKED_FROM:
            return False
        lib = self._seq_lib()
        key = ("chunked_retention", dk, dv, rot_dims, q.stride(0), k.stride(0), v.stride(0))
        ok = self._routes.get(key)
        if ok is None:
            ok = self._routes[key] = int(lib.sb_chunked_retention_supports(dk, dv, rot_dims, q.stride(0), k.stride(0), v.stride(0)))
        if not ok or any(x.data_ptr() % 8 for x in (q, k, v)):
            return False
        rows, n_list, chunks = None, shape.rows, q.shape[0] // 64 + shape.rows
        neg_q = getattr(shape, "neg_q_sorted", None)
        if neg_q is not None and getattr(shape, "rows_by_q", None) is not None:
            n_list = bisect.bisect_left(neg_q, -self.CHUNKED_FROM)
            rows, chunks = shape.rows_by_q, sum(-(n // 64) for n in neg_q[:n_list])
        if n_list * heads > 65535:
            return False
        angles = None
        if rot_dims:
            # one table for all layers with these frequencies: it depends on the step's positions alone
            memo_key = ("angle_table", inv_freq.data_ptr(), rot_dims)
            angles = ctx.memo.get(memo_key)
            if angles is None:
                angles = ctx.memo[memo_key] = torch.empty((q.shape[0], rot_dims // 2, 2), dtype=torch.float32, device=q.device)
                self.launches += 1
                _check(lib.sb_angle_table(_p(ctx.positions), _p(inv_freq), rot_dims // 2, q.shape[0], _p(angles), self._s()), "angle table")
        sums = torch.empty((chunks, heads, dk, dv), dtype=torch.float32, device=q.device)
        self.launches += 3
        _check(lib.sb_chunked_retention(
            _p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(angles), int(rot_dims), ctypes.c_float(k_scale), _p(decay), _p(state),
            ctypes.c_longlong(state.stride(0)), _p(ctx.slots), _p(ctx.cu_q), _p(rows), n_list, shape.max_q, self.CHUNKED_FROM, _p(out),
            out.stride(0), heads, dk, dv, _p(sums), self._s()), "chunked retention")
        return True

    def gated_norm(self, y, out, groups: int = 0, eps: float = 0.0, weight=None, gate=None, gate_act: str = "sigmoid",
                   gate_first: bool = False, scale: float = 1.0) -> None:
        """out = scale * [gate *] rms_groups([gate *] y) * weight: y float [T, C]; ``groups`` equal parts of a row are each divided
        by their root mean square (0: no division); y is float or of out's type; weight [w] with w dividing C; gate [T, g] with g dividing C."""
        self.launches += 1
        _check(self._seq_lib().sb_gated_norm(
            _p(y), _DT[y.dtype], y.stride(0), _p(gate), gate.stride(0) if gate is not None else 0, gate.shape[1] if gate is not None else 0,
            {"sigmoid": 0, "silu": 1}[gate_act], 1 if gate_first else 0, _p(weight), _DT[weight.dtype] if weight is not None else 0,
            weight.shape[0] if weight is not None else 0, _p(out), out.stride(0), y.shape[0], y.shape[1], groups, ctypes.c_float(eps),
            ctypes.c_float(scale), _DT[out.dtype], self._s()), "norm and gate")

    def kv_norm_cache_write(self, qkv, positions, token_row, heads, kv_heads, head_dim, norm_dim, eps, k_cache, v_cache, block_table,
                            page_size) -> None:
        """Keys and values of the step's tokens into their pages, without rotation; with norm_dim > 0 each value head is first
        divided by the root mean square of its first norm_dim elements."""
        self.launches += 1
        _check(self._seq_lib().sb_kv_norm_cache_write(
            _p(qkv), qkv.stride(0), _p(positions), _p(token_row), heads, kv_heads, head_dim, norm_dim, ctypes.c_float(eps), _p(k_cache),
            _p(v_cache), _p(block_table), block_table.shape[1], page_size, k_cache.shape[0], qkv.shape[0], _p(self.errors_tensor()),
            _DT[qkv.dtype], self._s()), "cache write with value norm")

    def routed_experts(self, h, logits, w_gate_up, w_down, top: int, out, score: str = "sigmoid", renormalise: bool = False,
                       scale_input: bool = True, activation: str = "clamped_swish", limit: float = 0.0, alpha: float = 1.702,
                       outputs=None, choice_bias=None, renormalise_eps: float = 0.0, shared=None, shared_gated: bool = False,
                       weight_scale: float = 1.0, groups: int = 1, keep_groups: int = 1) -> None:
        """out[t] = sum over the ``top`` best experts e of expert_e(w_e * h[t]) (or w_e * expert_e(h[t])): logits float [T, E],
        w_gate_up [E, 2 ff, K], w_down [E, N, ff]. More: the router scores the first ``outputs`` columns of logits, of which those
        beyond the E experts stand for the token's input itself; ``choice_bias`` (float [outputs]) joins the scores for the choice
        only; ``renormalise_eps`` joins the sum the weights are divided by; ``shared`` [T, N] is added for every token, times
        sigmoid(logits[:, outputs]) if ``shared_gated``; every weight is multiplied by ``weight_scale``; only outputs of the
        ``keep_groups`` best of ``groups`` equal groups of neighbours can be chosen (a group is as good as its best output)."""
        lib = self._moe_lib()
        t = logits.shape[0]
        e = w_down.shape[0]
        more = outputs is not None
        if not more and logits.shape[1] != e:
            raise KernelError("routed_experts: one router logit per expert")
        if more and (scale_input or outputs < e or logits.shape[1] < outputs + (1 if shared_gated else 0)
                     or (outputs > e and w_down.shape[1] != h.shape[1])):
            raise KernelError("routed_experts: identity experts, a choice bias and a shared expert come with weights on the outputs")
        ff, n, k = w_down.shape[2], w_down.shape[1], h.shape[1]
        pairs = t * top
        dev = h.device
        tile_rows = lib.sb_moe_tile_rows(_DT[h.dtype], k, ff, h.stride(0))     # 64 on the tensor-core kernels, else 32
        max_tiles = pairs // tile_rows + min(e, pairs)
        ints = torch.empty(2 * pairs + e + 1 + 2 * max_tiles + 1, dtype=torch.int32, device=dev)
        idx, order = ints[:pairs], ints[pairs: 2 * pairs]
        offsets = ints[2 * pairs: 2 * pairs + e + 1]
        tiles = ints[2 * pairs + e + 1: 2 * pairs + e + 1 + 2 * max_tiles]
        n_tiles = ints[-1:]
        wts = torch.empty(pairs, dtype=torch.float32, device=dev)
        s = self._s()
        self.launches += 4
        if more:
            _check(lib.sb_moe_route_bias(_p(logits), logits.stride(0), outputs, top, {"sigmoid": 0, "softmax": 1}[score],
                                         1 if renormalise else 0, ctypes.c_float(renormalise_eps), _p(choice_bias), t, _p(idx), _p(wts),
                                         ctypes.c_float(weight_scale), int(groups), int(keep_groups), s), "expert choice")
        else:
            _check(lib.sb_moe_route(_p(logits), e, top, {"sigmoid": 0, "softmax": 1}[score], 1 if renormalise else 0, t, _p(idx), _p(wts), s),
                   "expert choice")
        _check(lib.sb_moe_sort(_p(idx), pairs, e, tile_rows, _p(offsets), _p(order), _p(tiles), _p(n_tiles), s), "grouping by expert")
        act = torch.empty((pairs, ff), dtype=h.dtype, device=dev)
        _check(lib.sb_moe_gate_up(_p(h), h.stride(0), _p(w_gate_up), _p(order), _p(offsets), _p(tiles), _p(n_tiles), _p(wts), top, pairs,
                                  e, k, ff, 1 if scale_input else 0, {"swiglu": 0, "clamped_swish": 1}[activation],
                                  ctypes.c_float(limit), ctypes.c_float(alpha), _p(act), _DT[h.dtype], s), "experts, gate and up")
        parts = out if (top == 1 and not more) else torch.empty((pairs, n), dtype=torch.float32, device=dev)
        _check(lib.sb_moe_down(_p(act), _p(w_down), _p(order), _p(offsets), _p(tiles), _p(n_tiles), _p(wts), pairs, e, ff, n,
                               0 if scale_input else 1, _p(parts), _DT[h.dtype], _DT[parts.dtype], tile_rows, s), "experts, down")
        if more:
            self.launches += 1
            gate = logits[:, outputs:] if shared_gated else None
            _check(lib.sb_moe_combine_more(_p(parts), _p(idx), _p(wts), e, _p(h), h.stride(0), _p(shared), _p(gate), logits.stride(0), top, t, n,
                                           _p(out), _DT[out.dtype], s), "sum over a token's experts, identity and shared expert")
        elif top > 1:
            self.launches += 1
            _check(lib.sb_moe_combine(_p(parts), top, t, n, _p(out), _DT[out.dtype], s), "sum over a token's experts")

    def table_experts(self, h, tokens, last_token, table, w_up, w_down, top: int, out, activation: str = "relu_squared") -> None:
        """out[t] = (1 / top) * sum over the experts e = table[token[t], :] of w_down[e] act(w_up[e] h[t]), act = relu squared:
        table int32 [vocab, top], w_up [E, ff, K], w_down [E, N, ff]. A token id -(s+1) stands for last_token[s]."""
        if activation != "relu_squared":
            raise KernelError(f"table_experts: activation {activation!r} is not known")
        lib = self._moe_lib()
        t = h.shape[0]
        e, ff, k = w_up.shape
        n = w_down.shape[1]
        pairs = t * top
        dev = h.device
        tile_rows = lib.sb_moe_tile_rows(_DT[h.dtype], k, ff, h.stride(0))
        max_tiles = pairs // tile_rows + min(e, pairs)
        ints = torch.empty(2 * pairs + e + 1 + 2 * max_tiles + 1, dtype=torch.int32, device=dev)
        idx, order = ints[:pairs], ints[pairs: 2 * pairs]
        offsets = ints[2 * pairs: 2 * pairs + e + 1]
        tiles = ints[2 * pairs + e + 1: 2 * pairs + e + 1 + 2 * max_tiles]
        n_tiles = ints[-1:]
        wts = torch.empty(pairs, dtype=torch.float32, device=dev)
        s = self._s()
        self.launches += 4
        _check(lib.sb_moe_route_table(_p(tokens), _p(last_token), last_token.shape[0] if last_token is not None else 0, _p(table),
                                      table.shape[0], e, top, t, _p(idx), _p(wts), _p(self.errors_tensor()), s), "expert choice by table")
        _check(lib.sb_moe_sort(_p(idx), pairs, e, tile_rows, _p(offsets), _p(order), _p(tiles), _p(n_tiles), s), "grouping by expert")
        act = torch.empty((pairs, ff), dtype=h.dtype, device=dev)
        _check(lib.sb_moe_up(_p(h), h.stride(0), _p(w_up), _p(order), _p(offsets), _p(tiles), _p(n_tiles), _p(wts), top, pairs, e, k, ff,
                             _p(act), _DT[h.dtype], s), "experts, up")
        parts = out if top == 1 else torch.empty((pairs, n), dtype=torch.float32, device=dev)
        _check(lib.sb_moe_down(_p(act), _p(w_down), _p(order), _p(offsets), _p(tiles), _p(n_tiles), _p(wts), pairs, e, ff, n, 1, _p(parts),
                               _DT[h.dtype], _DT[parts.dtype], tile_rows, s), "experts, down")
        if top > 1:
            self.launches += 1
            _check(lib.sb_moe_combine(_p(parts), top, t, n, _p(out), _DT[out.dtype], s), "sum over a token's experts")

    def sample(self, logits, temperature, req_ids, tok_index, seed, out, slots=None, last_token=None) -> None:
        self.launches += 1
        n = logits.shape[0]
        if self._sample_work is None or self._sample_work.numel() < 3 * n:
            # n 64-bit keys and n counters, zero now and after every call (kept alive for captured graphs)
            self._sample_work = torch.zeros(3 * max(n, 256), dtype=torch.int32, device=self.device)
            self._keep.append(self._sample_work)
        _check(self._core.sb_sample(_p(logits), _p(temperature), _p(req_ids), _p(tok_index), ctypes.c_ulonglong(seed),
                                    n, logits.shape[1], _p(out), _p(self._sample_work), _p(slots), _p(last_token), self._s()),
               "sample")


_INSTANCES: Dict[str, CudaKernels] = {}


def load_kernels(device="cuda:0", head_dims=(), verbose: bool = True) -> CudaKernels:
    """The kernels for ``device`` (one object per device; more head sizes are built when first used)."""
    if not torch.cuda.is_available():
        raise KernelError("no CUDA device is available: this engine has no CPU path")
    key = str(torch.device(device))
    k = _INSTANCES.get(key)
    if k is None:
        k = _INSTANCES[key] = CudaKernels(device, head_dims, verbose)
    else:
        for d in head_dims:
            k._attention_lib(d)
    return k
