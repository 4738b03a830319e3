"""ctypes access to liblitnice_backend_b200.so.

Two thin layers over the C ABI declared in include/litnice_backend_b200.h:

* ``Backend`` drives the litnicelm plugin table (BackendApiV1) the way the
  reference's DynamicLibraryBackend does (src/model/backend/device_backend.cpp:
  180-654): create(GPU), alloc, host<->device copies, one call per operator with
  byte-strided views. It works with any library exporting
  ``litnice_backend_get_api`` (the reference CPU plugin included), which is how
  the tests compare two plugins on identical views.
* ``Session`` drives the native token loop (litnice_b200_*).

There is no fallback: if the shared library is missing or no CUDA device is
present, construction raises.
"""
from __future__ import annotations

import ctypes as C
import os
from dataclasses import dataclass
from typing import Optional, Sequence, Tuple

import numpy as np

from .formats import ModelDims

HERE = os.path.dirname(os.path.abspath(__file__))
LIB_PATH = os.path.join(HERE, "liblitnice_backend_b200.so")
MAX_RANK = 6


class BackendTensorView(C.Structure):
    _fields_ = [("device", C.c_uint32), ("dtype", C.c_uint32), ("data", C.c_void_p),
                ("rank", C.c_uint32), ("rows", C.c_int64), ("cols", C.c_int64),
                ("stride_r_bytes", C.c_int64), ("stride_c_bytes", C.c_int64),
                ("dims", C.c_int64 * MAX_RANK), ("strides_bytes", C.c_int64 * MAX_RANK)]


class BackendMemoryInfo(C.Structure):
    _fields_ = [("available", C.c_uint32), ("free_bytes", C.c_uint64), ("total_bytes", C.c_uint64)]


_V = C.POINTER(BackendTensorView)
_H = C.c_void_p


def _fn(res, *args):
    return C.CFUNCTYPE(res, *args)


# Order of backend_plugin_api.hpp:26-162.
_API_FIELDS = [
    ("abi_version", C.c_uint32),
    ("create", _fn(C.c_void_p, C.c_uint32)),
    ("destroy", _fn(None, _H)),
    ("device", _fn(C.c_uint32, _H)),
    ("alloc", _fn(C.c_void_p, _H, C.c_uint64, C.c_uint32)),
    ("free", _fn(None, _H, C.c_void_p)),
    ("copy_host2device", _fn(None, _H, C.c_void_p, C.c_void_p, C.c_uint64)),
    ("copy_device2host", _fn(None, _H, C.c_void_p, C.c_void_p, C.c_uint64)),
    ("copy", _fn(None, _H, _V, _V)),
    ("fill", _fn(None, _H, _V, C.c_float)),
    ("add", _fn(None, _H, _V, _V, _V)),
    ("add_inplace", _fn(None, _H, _V, _V)),
    ("add_bias_rowwise", _fn(None, _H, _V, _V, _V)),
    ("add_bias_relu_rowwise", _fn(None, _H, _V, _V, _V)),
    ("add_bias_relu_rowwise_inplace", _fn(None, _H, _V, _V)),
    ("mul_scalar", _fn(None, _H, _V, C.c_float, _V)),
    ("sum_squares_f32", _fn(C.c_float, _H, _V)),
    ("relu", _fn(None, _H, _V, _V)),
    ("relu_backward", _fn(None, _H, _V, _V, _V)),
    ("relu_backward_inplace", _fn(None, _H, _V, _V)),
    ("row_sum", _fn(None, _H, _V, _V)),
    ("gemm", _fn(None, _H, _V, _V, _V)),
    ("gemm_ranked_matrix_rhs", _fn(None, _H, _V, _V, _V)),
    ("gemm_ranked_matrix_rhs_t", _fn(None, _H, _V, _V, _V)),
    ("gemm_ranked_reduce_lhs_t", _fn(None, _H, _V, _V, _V)),
    ("gemm_batched", _fn(None, _H, _V, _V, _V)),
    ("gemm_batched_lhs_t", _fn(None, _H, _V, _V, _V)),
    ("gemm_batched_rhs_t", _fn(None, _H, _V, _V, _V)),
    ("transpose", _fn(None, _H, _V, _V)),
    ("layernorm_forward", _fn(None, _H, _V, _V, _V, _V)),
    ("layernorm_backward", _fn(None, _H, _V, _V, _V, _V, _V, _V)),
    ("embedding_lookup", _fn(None, _H, _V, _V, _V)),
    ("accumulate_embedding_grads", _fn(None, _H, _V, _V, _V, _V)),
    ("cross_entropy_mean", _fn(None, _H, _V, _V, _V)),
    ("cross_entropy_mean_backward_inplace", _fn(None, _H, _V, _V, _V)),
    ("read_scalar_f32", _fn(C.c_float, _H, _V)),
    ("backward_from_logits_targets", _fn(None, _H, _V, _V)),
    ("softmax_rows", _fn(None, _H, _V, _V)),
    ("softmax_backward_rows", _fn(None, _H, _V, _V, _V)),
    ("scaled_causal_softmax_rows", _fn(None, _H, _V, C.c_float, _V)),
    ("supports_exec_context_iteration", _fn(C.c_uint32, _H)),
    ("start_exec_context_iteration", _fn(None, _H)),
    ("finish_exec_context_iteration", _fn(None, _H)),
    ("start_exec_context_group", _fn(None, _H)),
    ("finish_exec_context_group", _fn(None, _H)),
    ("gemm_batched_exec_context", _fn(None, _H, _V, _V, _V)),
    ("gemm_batched_lhs_t_exec_context", _fn(None, _H, _V, _V, _V)),
    ("gemm_batched_rhs_t_exec_context", _fn(None, _H, _V, _V, _V)),
    ("scaled_causal_softmax_rows_exec_context", _fn(None, _H, _V, C.c_float, _V)),
    ("softmax_backward_causal_rows_exec_context", _fn(None, _H, _V, _V, _V)),
    ("softmax_backward_causal_rows", _fn(None, _H, _V, _V, _V)),
    ("apply_causal_mask_inplace", _fn(None, _H, _V, C.c_float)),
    ("adamw_step", _fn(None, _H, _V, _V, _V, _V, C.c_uint64, C.c_float, C.c_float, C.c_float,
                       C.c_float, C.c_uint32)),
    ("is_file2device_read_supported", _fn(C.c_uint32, _H)),
    ("read_file2device", _fn(None, _H, C.c_char_p, C.c_void_p, C.c_uint64, C.c_uint64)),
    ("memory_info", _fn(BackendMemoryInfo, _H)),
]


class BackendApiV1(C.Structure):
    _fields_ = _API_FIELDS


API_ENTRY_NAMES = [name for name, _ in _API_FIELDS[1:]]

# What a host of the native loop binds (the diagnostics of the header's third section are
# left out on purpose).
NATIVE_SYMBOLS = [
    "litnice_b200_session_create", "litnice_b200_session_create_on", "litnice_b200_session_destroy",
    "litnice_b200_last_error",
    "litnice_b200_load_params", "litnice_b200_load_checkpoint", "litnice_b200_generate",
    "litnice_b200_upload_prompts", "litnice_b200_run", "litnice_b200_download_tokens",
    "litnice_b200_keep_step_logits", "litnice_b200_read_step_logits", "litnice_b200_forward",
    "litnice_b200_inspect", "litnice_b200_sample_logits", "litnice_b200_get_stats",
    "litnice_b200_gemv_noalloc",
    "litnice_b200_session_create_model", "litnice_b200_architectures", "litnice_b200_model_dims",
    "litnice_b200_extend", "litnice_b200_release",
]


def load_library(path: Optional[str] = None) -> C.CDLL:
    path = path or LIB_PATH
    if not os.path.exists(path):
        raise RuntimeError(f"{path} is missing: build it with `make -C litnicelm_b200/csrc` "
                           "(there is no CPU fallback)")
    return C.CDLL(path)


def get_api(lib: C.CDLL) -> BackendApiV1:
    lib.litnice_backend_get_api.restype = C.POINTER(BackendApiV1)
    api = lib.litnice_backend_get_api()
    if not api or api.contents.abi_version != 16:
        raise RuntimeError("backend ABI mismatch")
    return api.contents


def projection_time(m: int, k: int, n: int, repeats: int = 20, engine: int = 1,
                    lib: Optional[C.CDLL] = None) -> float:
    """Average device time in microseconds of one C[m,n] = A[m,k]·W[k,n] on the
    tensor-core (engine 1) or SIMT (engine 0) projection kernel, warm, launched
    back to back (litnice_b200_projection_time)."""
    lib = lib or load_library()
    f32p = C.POINTER(C.c_float)
    fn = lib.litnice_b200_projection_time
    fn.argtypes = [C.c_int32, f32p, C.c_int32, C.c_int32, f32p, C.c_int32, f32p, C.c_int32, C.POINTER(C.c_double)]
    fn.restype = C.c_int
    rng = np.random.default_rng(0)
    a = rng.standard_normal((m, k), dtype=np.float32)
    w = (rng.standard_normal((k, n), dtype=np.float32) * 0.02).astype(np.float32)
    c = np.empty((m, n), np.float32)
    us = C.c_double(0)
    rc = fn(engine, a.ctypes.data_as(f32p), m, k, w.ctypes.data_as(f32p), n, c.ctypes.data_as(f32p), repeats,
            C.byref(us))
    if rc != 0:
        raise RuntimeError(f"litnice_b200_projection_time failed with status {rc}")
    return us.value


def gemv_host(x: np.ndarray, w: np.ndarray, bias: Optional[np.ndarray] = None,
              residual: Optional[np.ndarray] = None, relu: bool = False,
              ln: Optional[Tuple[np.ndarray, np.ndarray]] = None,
              lib: Optional[C.CDLL] = None) -> np.ndarray:
    """out[m, n] = x[m, k] . W[k, n] (+ bias) (+ residual) (ReLU) for m <= 8 on the few-row
    kernels of the output head (litnice_b200_gemv_host: host buffers in, host buffer out)."""
    lib = lib or load_library()
    f32p = C.POINTER(C.c_float)
    fn = lib.litnice_b200_gemv_host
    fn.argtypes = [f32p, C.c_int32, f32p, C.c_int32, C.c_int32, f32p, f32p, C.c_int32, f32p, f32p, f32p]
    fn.restype = C.c_int
    x = np.ascontiguousarray(x, np.float32)
    w = np.ascontiguousarray(w, np.float32)
    m, k = x.shape
    n = w.shape[1]
    out = np.empty((m, n), np.float32)
    b = None
    if bias is not None:
        bias = np.ascontiguousarray(bias, np.float32).ravel()
        b = bias.ctypes.data_as(f32p)
    r = None
    if residual is not None:
        residual = np.ascontiguousarray(residual, np.float32)
        r = residual.ctypes.data_as(f32p)
    g = be = None
    if ln is not None:   # (gamma, beta): the rows of x pass through LayerNorm inside the kernel
        gamma = np.ascontiguousarray(ln[0], np.float32).ravel()
        beta = np.ascontiguousarray(ln[1], np.float32).ravel()
        g, be = gamma.ctypes.data_as(f32p), beta.ctypes.data_as(f32p)
    rc = fn(x.ctypes.data_as(f32p), m, w.ctypes.data_as(f32p), k, n, b, r, 1 if relu else 0, g, be,
            out.ctypes.data_as(f32p))
    if rc != 0:
        raise RuntimeError(f"litnice_b200_gemv_host failed with status {rc}")
    return out


def gemv_time(m: int, k: int, n: int, repeats: int = 50, cold_l2: int = 2, force_tn: int = 0,
              force_splits: int = 0, lib: Optional[C.CDLL] = None) -> Tuple[float, int]:
    """(mean device microseconds, kernels per call) of the few-row product. cold_l2 = 2:
    `repeats` calls back to back between one pair of CUDA events, each on the next of a
    ring of weight copies larger than three times the L2 (every call reads HBM);
    1: events around each call, a 256 MB buffer written before it; 0: the same matrix
    every call (L2-resident when it fits)."""
    lib = lib or load_library()
    fn = lib.litnice_b200_gemv_time
    fn.argtypes = [C.c_int32] * 7 + [C.POINTER(C.c_double), C.POINTER(C.c_int32)]
    fn.restype = C.c_int
    us, nl = C.c_double(0), C.c_int32(0)
    rc = fn(m, k, n, repeats, int(cold_l2), force_tn, force_splits, C.byref(us), C.byref(nl))
    if rc != 0:
        raise RuntimeError(f"litnice_b200_gemv_time failed with status {rc}")
    return us.value, nl.value


@dataclass
class DevTensor:
    """A byte-strided view into plugin-allocated memory (TensorView of the
    reference, src/model/tensor.hpp:121-323)."""
    ptr: int
    shape: Tuple[int, ...]
    strides: Tuple[int, ...]  # bytes
    dtype: int = 0            # 0 f32, 1 i32
    device: int = 1

    def view(self) -> BackendTensorView:
        v = BackendTensorView()
        v.device, v.dtype, v.data, v.rank = self.device, self.dtype, self.ptr, len(self.shape)
        v.rows = self.shape[0]
        v.cols = self.shape[1] if len(self.shape) > 1 else 0
        v.stride_r_bytes = self.strides[-2] if len(self.shape) >= 2 else 0
        v.stride_c_bytes = self.strides[-1]
        for i, (d, s) in enumerate(zip(self.shape, self.strides)):
            v.dims[i], v.strides_bytes[i] = d, s
        return v


class Backend:
    """One plugin instance, driven as the reference host drives it."""

    def __init__(self, lib_path: Optional[str] = None, device_kinds: Sequence[int] = (1, 0)):
        self.lib = load_library(lib_path)
        self.api = get_api(self.lib)
        self.h = None
        for kind in device_kinds:  # device_backend.cpp:208-220
            self.h = self.api.create(kind)
            if self.h:
                break
        if not self.h:
            raise RuntimeError("backend create failed")
        self.device = int(self.api.device(self.h))
        self._allocs = []

    def close(self):
        if self.h:
            for p in self._allocs:
                self.api.free(self.h, p)
            self._allocs = []
            self.api.destroy(self.h)
            self.h = None

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()

    def alloc(self, nbytes: int, alignment: int = 64) -> int:
        p = self.api.alloc(self.h, nbytes, alignment)
        if not p:
            raise MemoryError("plugin alloc returned null")
        self._allocs.append(p)
        return int(p)

    def upload(self, ptr: int, arr: np.ndarray, offset: int = 0):
        arr = np.ascontiguousarray(arr)
        self.api.copy_host2device(self.h, ptr + offset, arr.ctypes.data, arr.nbytes)

    def download(self, ptr: int, nbytes: int, offset: int = 0) -> np.ndarray:
        out = np.empty(nbytes, dtype=np.uint8)
        self.api.copy_device2host(self.h, out.ctypes.data, ptr + offset, nbytes)
        return out

    def put(self, buffer_ptr: int, t: DevTensor, values: np.ndarray, buffer_bytes: int):
        """Scatter `values` (logical shape of t) into the strided view t by
        rewriting the whole backing buffer from the host."""
        host = self.download(buffer_ptr, buffer_bytes)
        dt = np.float32 if t.dtype == 0 else np.int32
        view = np.lib.stride_tricks.as_strided(
            host[t.ptr - buffer_ptr:].view(dt), shape=t.shape, strides=t.strides, writeable=True)
        view[...] = values
        self.upload(buffer_ptr, host)

    def get(self, buffer_ptr: int, t: DevTensor, buffer_bytes: int) -> np.ndarray:
        host = self.download(buffer_ptr, buffer_bytes)
        dt = np.float32 if t.dtype == 0 else np.int32
        return np.lib.stride_tricks.as_strided(host[t.ptr - buffer_ptr:].view(dt), shape=t.shape,
                                               strides=t.strides).copy()

    def call(self, name: str, *args):
        """Invoke a table entry; DevTensor arguments become view pointers."""
        conv = []
        keep = []
        for a in args:
            if isinstance(a, DevTensor):
                v = a.view()
                keep.append(v)
                conv.append(C.byref(v))
            else:
                conv.append(a)
        return getattr(self.api, name)(self.h, *conv)


class B200Dims(C.Structure):
    _fields_ = [("n_layers", C.c_int32), ("n_heads", C.c_int32), ("d_model", C.c_int32),
                ("d_ff", C.c_int32), ("vocab_size", C.c_int32), ("max_seq_len", C.c_int32),
                ("alignment_bytes", C.c_uint64)]


class B200Sampling(C.Structure):
    _fields_ = [("temp", C.c_float), ("top_k", C.c_uint32), ("top_p", C.c_float)]


class B200Stats(C.Structure):
    _fields_ = [("device_ms", C.c_double), ("kernel_launches", C.c_int64), ("tokens", C.c_int64),
                ("h2d_bytes", C.c_int64), ("d2h_bytes", C.c_int64), ("gemm_ms", C.c_double),
                ("gemm_launches", C.c_int64), ("gemm_flops", C.c_double), ("attn_ms", C.c_double),
                ("attn_launches", C.c_int64), ("gemm_span_ms", C.c_double), ("gemm_span_launches", C.c_int64),
                ("gemm_span_flops", C.c_double), ("attn_span_ms", C.c_double), ("attn_span_launches", C.c_int64),
                ("step_span_ms", C.c_double)]


class NativeError(RuntimeError):
    pass


class Session:
    """Native token loop: generate_text of the reference (inference.cpp:265-296)
    for n independent streams in lockstep, entirely on the GPU."""

    def _bind(self, lib_path: Optional[str]):
        self.lib = load_library(lib_path)
        L = self.lib
        i32p, f32p, u32p = C.POINTER(C.c_int32), C.POINTER(C.c_float), C.POINTER(C.c_uint32)
        L.litnice_b200_session_create.argtypes = [C.POINTER(B200Dims), C.c_int32, C.POINTER(C.c_void_p)]
        L.litnice_b200_session_destroy.argtypes = [C.c_void_p]
        L.litnice_b200_session_destroy.restype = None
        L.litnice_b200_last_error.argtypes = [C.c_void_p]
        L.litnice_b200_last_error.restype = C.c_char_p
        L.litnice_b200_load_params.argtypes = [C.c_void_p, C.c_void_p, C.c_uint64]
        L.litnice_b200_load_checkpoint.argtypes = [C.c_void_p, C.c_char_p]
        L.litnice_b200_generate.argtypes = [C.c_void_p, i32p, C.c_int32, C.c_int32, C.c_int32,
                                            C.POINTER(B200Sampling), u32p, i32p, i32p]
        L.litnice_b200_upload_prompts.argtypes = [C.c_void_p, i32p, C.c_int32, C.c_int32, u32p]
        L.litnice_b200_run.argtypes = [C.c_void_p, C.c_int32, C.POINTER(B200Sampling), i32p]
        L.litnice_b200_download_tokens.argtypes = [C.c_void_p, i32p, C.c_int32]
        L.litnice_b200_keep_step_logits.argtypes = [C.c_void_p, C.c_int32]
        L.litnice_b200_read_step_logits.argtypes = [C.c_void_p, f32p, C.c_int64]
        L.litnice_b200_forward.argtypes = [C.c_void_p, i32p, C.c_int32, C.c_int32, C.c_int32, f32p]
        L.litnice_b200_inspect.argtypes = [C.c_void_p, i32p, C.c_int32, C.c_int32, f32p]
        L.litnice_b200_sample_logits.argtypes = [C.c_void_p, f32p, C.c_int32, C.POINTER(B200Sampling),
                                                 u32p, C.c_int32, i32p]
        L.litnice_b200_get_stats.argtypes = [C.c_void_p, C.POINTER(B200Stats)]
        L.litnice_b200_profile_step.argtypes = [C.c_void_p, C.c_int32, C.c_int32, C.c_int32]
        L.litnice_b200_session_create_model.argtypes = [C.c_char_p, C.c_int32, C.c_int32, C.c_int32,
                                                        C.POINTER(C.c_void_p)]
        L.litnice_b200_model_dims.argtypes = [C.c_void_p, C.POINTER(B200Dims)]
        L.litnice_b200_extend.argtypes = [C.c_void_p, C.c_int32, i32p, C.c_int32, i32p, C.c_int32, f32p]
        L.litnice_b200_release.argtypes = [C.c_void_p, C.c_int32]
        return L

    def __init__(self, dims: ModelDims, max_streams: int = 1, lib_path: Optional[str] = None,
                 device: Optional[int] = None):
        L = self._bind(lib_path)
        self.dims = dims
        self.max_streams = max_streams
        cd = B200Dims(dims.n_layers, dims.n_heads, dims.d_model, dims.d_ff, dims.vocab, dims.max_seq,
                      dims.alignment)
        self.h = C.c_void_p()
        if device is None:
            rc = L.litnice_b200_session_create(C.byref(cd), max_streams, C.byref(self.h))
        else:
            L.litnice_b200_session_create_on.argtypes = [C.POINTER(B200Dims), C.c_int32, C.c_int32,
                                                         C.POINTER(C.c_void_p)]
            rc = L.litnice_b200_session_create_on(C.byref(cd), max_streams, device, C.byref(self.h))
        if rc != 0:
            msg = L.litnice_b200_last_error(self.h).decode() if self.h else "no session"
            if self.h:
                L.litnice_b200_session_destroy(self.h)
                self.h = None
            raise NativeError(f"session_create failed ({rc}): {msg}")

    def close(self):
        if self.h:
            self.lib.litnice_b200_session_destroy(self.h)
            self.h = None

    def __enter__(self):
        return self

    def __exit__(self, *exc):
        self.close()

    def _check(self, rc: int, what: str):
        if rc != 0:
            raise NativeError(f"{what} failed ({rc}): {self.lib.litnice_b200_last_error(self.h).decode()}")

    @staticmethod
    def _i32(a):
        return a.ctypes.data_as(C.POINTER(C.c_int32))

    @staticmethod
    def _f32(a):
        return a.ctypes.data_as(C.POINTER(C.c_float))

    def load_params(self, arena: np.ndarray):
        arena = np.ascontiguousarray(arena)
        self._check(self.lib.litnice_b200_load_params(self.h, arena.ctypes.data, arena.nbytes), "load_params")

    def load_checkpoint(self, path: str):
        self._check(self.lib.litnice_b200_load_checkpoint(self.h, path.encode()), "load_checkpoint")

    def keep_step_logits(self, enable: bool):
        self._check(self.lib.litnice_b200_keep_step_logits(self.h, 1 if enable else 0), "keep_step_logits")

    def _seeds(self, seeds, n):
        if seeds is None:
            return None, None
        arr = np.ascontiguousarray(seeds, dtype=np.uint32)
        assert arr.shape == (n,)
        return arr, arr.ctypes.data_as(C.POINTER(C.c_uint32))

    def generate(self, prompts: np.ndarray, max_new: int, temp: float = 0.0, top_k: int = 0,
                 top_p: float = 1.0, seeds=None) -> np.ndarray:
        """prompts [n_streams, prompt_len] int32 -> tokens [n_streams, produced]."""
        prompts = np.ascontiguousarray(prompts, dtype=np.int32)
        if prompts.ndim == 1:
            prompts = prompts[None, :]
        n, plen = prompts.shape
        out = np.zeros((n, max(1, max_new)), dtype=np.int32)
        count = C.c_int32(0)
        sp = B200Sampling(temp, top_k, top_p)
        keep, sptr = self._seeds(seeds, n)
        self._check(self.lib.litnice_b200_generate(self.h, self._i32(prompts), n, plen, max_new,
                                                   C.byref(sp), sptr, self._i32(out), C.byref(count)),
                    "generate")
        return out[:, :count.value].copy()

    def upload_prompts(self, prompts: np.ndarray, seeds=None):
        prompts = np.ascontiguousarray(prompts, dtype=np.int32)
        if prompts.ndim == 1:
            prompts = prompts[None, :]
        n, plen = prompts.shape
        keep, sptr = self._seeds(seeds, n)
        self._check(self.lib.litnice_b200_upload_prompts(self.h, self._i32(prompts), n, plen, sptr),
                    "upload_prompts")
        self._n = n

    def run(self, max_new: int, temp: float = 0.0, top_k: int = 0, top_p: float = 1.0) -> int:
        sp = B200Sampling(temp, top_k, top_p)
        count = C.c_int32(0)
        self._check(self.lib.litnice_b200_run(self.h, max_new, C.byref(sp), C.byref(count)), "run")
        return count.value

    def download_tokens(self, count: int) -> np.ndarray:
        out = np.zeros((self._n, max(1, count)), dtype=np.int32)
        self._check(self.lib.litnice_b200_download_tokens(self.h, self._i32(out), max(1, count)),
                    "download_tokens")
        return out[:, :count]

    def read_step_logits(self, steps: int, n_streams: int) -> np.ndarray:
        out = np.empty((steps, n_streams, self.dims.vocab), dtype=np.float32)
        self._check(self.lib.litnice_b200_read_step_logits(self.h, self._f32(out), out.size), "read_step_logits")
        return out

    def forward(self, ids: np.ndarray, all_rows: bool = False) -> np.ndarray:
        ids = np.ascontiguousarray(ids, dtype=np.int32)
        if ids.ndim == 1:
            ids = ids[None, :]
        n, s = ids.shape
        out = np.empty((n, s, self.dims.vocab) if all_rows else (n, self.dims.vocab), dtype=np.float32)
        self._check(self.lib.litnice_b200_forward(self.h, self._i32(ids), n, s, 1 if all_rows else 0,
                                                  self._f32(out)), "forward")
        return out

    def inspect(self, ids: np.ndarray) -> np.ndarray:
        ids = np.ascontiguousarray(ids, dtype=np.int32)
        if ids.ndim == 1:
            ids = ids[None, :]
        n, s = ids.shape
        out = np.empty((n, self.dims.vocab), dtype=np.float32)
        self._check(self.lib.litnice_b200_inspect(self.h, self._i32(ids), n, s, self._f32(out)), "inspect")
        return out

    def sample_logits(self, logits: np.ndarray, temp: float, top_k: int, top_p: float, seeds,
                      draws: int = 1) -> np.ndarray:
        logits = np.ascontiguousarray(logits, dtype=np.float32)
        n = logits.shape[0]
        out = np.empty((n, draws), dtype=np.int32)
        sp = B200Sampling(temp, top_k, top_p)
        keep, sptr = self._seeds(seeds, n)
        self._check(self.lib.litnice_b200_sample_logits(self.h, self._f32(logits), n, C.byref(sp), sptr,
                                                        draws, self._i32(out)), "sample_logits")
        return out

    def stats(self) -> B200Stats:
        st = B200Stats()
        self._check(self.lib.litnice_b200_get_stats(self.h, C.byref(st)), "get_stats")
        return st

    def profile_step(self, n_streams: int, seq_len: int, repeats: int = 3) -> B200Stats:
        self._check(self.lib.litnice_b200_profile_step(self.h, n_streams, seq_len, repeats), "profile_step")
        return self.stats()


DTYPES = {"bfloat16": 0, "float32": 1}


def architectures(lib_path: Optional[str] = None) -> list:
    """Names of the decoder designs the library serves from a model folder."""
    lib = load_library(lib_path)
    lib.litnice_b200_architectures.restype = C.c_char_p
    return lib.litnice_b200_architectures().decode().split(",")


class ModelSession(Session):
    """The native loop on a model folder (config.json + model.safetensors) of a registered
    design: everything a Session does on the slots' caches and state, plus ``extend`` and
    ``release`` for sequences fed in portions."""

    def __init__(self, model_dir: str, dtype: str = "bfloat16", max_streams: int = 1,
                 lib_path: Optional[str] = None, device: int = -1):
        L = self._bind(lib_path)
        self.max_streams = max_streams
        self.h = C.c_void_p()
        rc = L.litnice_b200_session_create_model(os.fspath(model_dir).encode(), DTYPES[dtype], max_streams, device,
                                                 C.byref(self.h))
        if rc != 0:
            msg = L.litnice_b200_last_error(self.h).decode()
            if self.h:
                L.litnice_b200_session_destroy(self.h)
                self.h = None
            raise NativeError(f"session_create_model failed ({rc}): {msg}")
        d = B200Dims()
        self._check(L.litnice_b200_model_dims(self.h, C.byref(d)), "model_dims")
        self.dims = ModelDims(d.n_layers, 1, d.d_model, 0, d.vocab_size, d.max_seq_len)

    def extend(self, slot: int, tokens, want=()) -> np.ndarray:
        """Appends tokens to the sequence in `slot`; logits [len(want), vocab] of the wanted places."""
        tokens = np.ascontiguousarray(tokens, dtype=np.int32)
        want = np.ascontiguousarray(want, dtype=np.int32)
        out = np.empty((len(want), self.dims.vocab), dtype=np.float32)
        self._check(self.lib.litnice_b200_extend(self.h, slot, self._i32(tokens), len(tokens), self._i32(want), len(want),
                                                 self._f32(out)), "extend")
        return out

    def release(self, slot: int):
        rc = self.lib.litnice_b200_release(self.h, slot)
        if rc != 0:
            raise NativeError(f"release failed ({rc})")


ACTIVATIONS = {None: 0, "gelu": 1, "gelu_tanh": 2}


def bf16_product_host(a: np.ndarray, w: np.ndarray, engine: int, n_half: int = 0, act: Optional[str] = None,
                      gated: bool = False, c: Optional[np.ndarray] = None, lib: Optional[C.CDLL] = None) -> np.ndarray:
    """c[m, n] = a[m, k] w[n, k]^T on bfloat16 operands (litnice_b200_bf16_product_host); c given: added to."""
    lib = lib or load_library()
    f32p = C.POINTER(C.c_float)
    fn = lib.litnice_b200_bf16_product_host
    fn.argtypes = [C.c_int32, f32p, C.c_int32, C.c_int32, f32p] + [C.c_int32] * 5 + [f32p]
    a, w = np.ascontiguousarray(a, np.float32), np.ascontiguousarray(w, np.float32)
    m, k = a.shape
    n = w.shape[0]
    out = np.zeros((m, n - n_half // 2 if gated else n), np.float32) if c is None else np.array(c, np.float32, order="C")
    p = lambda x: x.ctypes.data_as(f32p)
    rc = fn(engine, p(a), m, k, p(w), n, n_half, ACTIVATIONS[act], int(gated), int(c is not None), p(out))
    if rc != 0:
        raise RuntimeError(f"litnice_b200_bf16_product_host failed with status {rc}")
    return out


def _floats(*arrays):
    """Contiguous float32 arrays and their pointers (None stays None)."""
    f32p = C.POINTER(C.c_float)
    held = [None if a is None else np.ascontiguousarray(a, np.float32) for a in arrays]
    return held, [None if a is None else a.ctypes.data_as(f32p) for a in held]


def residual_norm_host(x: np.ndarray, y: Optional[np.ndarray], after: Optional[np.ndarray], before: Optional[np.ndarray],
                       base: float, eps: float, dtype: str = "float32", lib: Optional[C.CDLL] = None):
    """(x + rms(y) (base + after), rms of that times (base + before) or None) (litnice_b200_residual_norm_host)."""
    lib = lib or load_library()
    f32p = C.POINTER(C.c_float)
    fn = lib.litnice_b200_residual_norm_host
    fn.argtypes = [C.c_int32] + [f32p] * 4 + [C.c_float, C.c_int32, C.c_int32, C.c_float, f32p]
    n, d = x.shape
    x = np.array(x, np.float32, order="C")
    h = None if before is None else np.empty((n, d), np.float32)
    held, p = _floats(x, y, after, before, h)
    rc = fn(DTYPES[dtype], p[0], p[1], p[2], p[3], base, n, d, eps, p[4])
    if rc != 0:
        raise RuntimeError(f"litnice_b200_residual_norm_host failed with status {rc}")
    return held[0], held[4]


def delta_host(rows: np.ndarray, ba: np.ndarray, conv: np.ndarray, a_log: np.ndarray, dt_bias: np.ndarray, norm: np.ndarray,
               eps: float, heads: int, groups: int, dim: int, vdim: int, portions: Optional[Sequence[int]] = None,
               dtype: str = "float32", lib: Optional[C.CDLL] = None):
    """rows [streams, n, q | k | v | gate], ba [streams, n, 2 * heads]: (outputs [streams, n, heads * vdim], final states
    [streams, heads, dim, vdim]) of the gated delta rule (litnice_b200_delta_host)."""
    lib = lib or load_library()
    f32p, i32p = C.POINTER(C.c_float), C.POINTER(C.c_int32)
    fn = lib.litnice_b200_delta_host
    fn.argtypes = [C.c_int32] + [f32p] * 6 + [C.c_float] + [C.c_int32] * 7 + [i32p, C.c_int32, f32p, f32p]
    b, n = rows.shape[:2]
    out, state = np.empty((b, n, heads * vdim), np.float32), np.empty((b, heads, dim, vdim), np.float32)
    por = np.ascontiguousarray([n] if portions is None else portions, np.int32)
    held, p = _floats(rows, ba, conv, a_log, dt_bias, norm, out, state)
    rc = fn(DTYPES[dtype], *p[:6], eps, b, n, heads, groups, dim, vdim, conv.shape[1], por.ctypes.data_as(i32p), len(por), p[6],
            p[7])
    if rc != 0:
        raise RuntimeError(f"litnice_b200_delta_host failed with status {rc}")
    return held[6], held[7]


SPANS = {"window": 0, "chunk": 1}


def grouped_attention_host(engine: int, rows: np.ndarray, n: int, q_weight: np.ndarray, k_weight: np.ndarray, eps: float,
                           turns: np.ndarray, amplitude: float, heads: int, groups: int, dim: int, vdim: int, scale: float,
                           span: str, size: int, lib: Optional[C.CDLL] = None):
    """rows [streams, T, q | k | v]: (rotated queries of the last n positions, rotated keys of all, outputs of the last n)
    (litnice_b200_grouped_attention_host)."""
    lib = lib or load_library()
    f32p, f64p = C.POINTER(C.c_float), C.POINTER(C.c_double)
    fn = lib.litnice_b200_grouped_attention_host
    fn.argtypes = ([C.c_int32] + [f32p] * 3 + [C.c_float, C.c_int32, f64p, C.c_float] + [C.c_int32] * 7 +
                   [C.c_float, C.c_int32, C.c_int32, f32p, f32p, f32p])
    b, t = rows.shape[:2]
    turns = np.ascontiguousarray(turns, np.float64)
    q, k = np.empty((b, n, heads * dim), np.float32), np.empty((b, t, groups * dim), np.float32)
    out = np.empty((b, n, heads * vdim), np.float32)
    held, p = _floats(rows, q_weight, k_weight, q, k, out)
    rc = fn(engine, *p[:3], eps, 2 * len(turns), turns.ctypes.data_as(f64p), amplitude, b, t - n, n, heads, groups, dim, vdim,
            scale, SPANS[span], size, *p[3:])
    if rc != 0:
        raise RuntimeError(f"litnice_b200_grouped_attention_host failed with status {rc}")
    return held[3], held[4], held[5]


def rms_canon_host(x: np.ndarray, gain: float, eps: float, w1: np.ndarray, w2: Optional[np.ndarray] = None,
                   portions: Optional[Sequence[int]] = None, dtype: str = "float32", lib: Optional[C.CDLL] = None):
    """(h + conv1(h), h + conv2(h) or None) with h the scalar-gain RMS norm of x (litnice_b200_rms_canon_host)."""
    lib = lib or load_library()
    f32p, i32p = C.POINTER(C.c_float), C.POINTER(C.c_int32)
    fn = lib.litnice_b200_rms_canon_host
    fn.argtypes = [C.c_int32, f32p, C.c_int32, C.c_int32, C.c_float, C.c_float, C.c_int32, f32p, f32p, i32p, C.c_int32,
                   f32p, f32p]
    x = np.ascontiguousarray(x, np.float32)
    n, d = x.shape
    w1 = np.ascontiguousarray(w1, np.float32)
    por = np.ascontiguousarray([n] if portions is None else portions, np.int32)
    o1 = np.empty((n, d), np.float32)
    p = lambda v: None if v is None else v.ctypes.data_as(f32p)
    o2 = None
    if w2 is not None:
        w2, o2 = np.ascontiguousarray(w2, np.float32), np.empty((n, d), np.float32)
    rc = fn(DTYPES[dtype], p(x), n, d, gain, eps, w1.shape[1], p(w1), p(w2), por.ctypes.data_as(i32p), len(por), p(o1), p(o2))
    if rc != 0:
        raise RuntimeError(f"litnice_b200_rms_canon_host failed with status {rc}")
    return o1, o2


def latent_attention_host(engine: int, q: np.ndarray, dkv: np.ndarray, gain: np.ndarray, eps: float, w_uk: np.ndarray,
                          w_uv: np.ndarray, heads: int, dim: int, vdim: int, scale: float, window: int,
                          lib: Optional[C.CDLL] = None) -> np.ndarray:
    """q [streams, n, heads * dim], dkv [streams, T, rank]: outputs of the last n positions
    (litnice_b200_latent_attention_host)."""
    lib = lib or load_library()
    f32p = C.POINTER(C.c_float)
    fn = lib.litnice_b200_latent_attention_host
    fn.argtypes = [C.c_int32, f32p, f32p, f32p, C.c_float, f32p, f32p] + [C.c_int32] * 7 + [C.c_float, C.c_int32, f32p]
    arrs = [np.ascontiguousarray(v, np.float32) for v in (q, dkv, gain, w_uk, w_uv)]
    q, dkv, gain, w_uk, w_uv = arrs
    b, n = q.shape[:2]
    t, rank = dkv.shape[1:]
    out = np.empty((b, n, heads * vdim), np.float32)
    p = lambda v: v.ctypes.data_as(f32p)
    rc = fn(engine, p(q), p(dkv), p(gain), eps, p(w_uk), p(w_uv), b, t - n, n, heads, dim, vdim, rank, scale, window, p(out))
    if rc != 0:
        raise RuntimeError(f"litnice_b200_latent_attention_host failed with status {rc}")
    return out
