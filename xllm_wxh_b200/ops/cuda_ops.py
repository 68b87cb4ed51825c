"""ctypes bindings of `libxllm_kernels.so` (hand-written sm_100a kernels; sources in `csrc/cuda`).

Kernels are launched on PyTorch's current stream, so they are captured by `torch.cuda.graph` like any other
work.  A missing or failing library raises: there is no silent fallback to PyTorch on a CUDA device.
"""
from __future__ import annotations

import ctypes
import os
from typing import Dict, Optional, Tuple

import torch

_HERE = os.path.dirname(os.path.abspath(__file__))
_LIB_PATH = os.environ.get("XLLM_KERNELS_SO") or os.path.join(os.path.dirname(_HERE), "libxllm_kernels.so")
_lib = None
launch_count = 0          # kernels launched through this module (reported by bench.py as `gpu_launches`)

c_void_p, c_int, c_long, c_float = ctypes.c_void_p, ctypes.c_int, ctypes.c_long, ctypes.c_float


class _TimedLib:
    """Opt-in profiling aid (`XLLM_KERNEL_TIMING=1`): brackets every kernel entry point with a pair of CUDA events on
    the current stream and accumulates device time per entry point.  Off by default; the events add a few
    microseconds of host time per launch, so numbers taken with it on are for shares, not for reporting."""
    _PLAIN = ("xl_dev_malloc", "xl_dev_free", "xl_ipc_get_handle", "xl_ipc_open_handle", "xl_ipc_close_handle",
              "xl_read_status", "xl_sm_count", "xl_gemm_force_bn", "xl_reset_status", "xl_prefill_use_tc", "xl_gemm_set_mode", "xl_gemm_pair_force_bn", "xl_gemm_pair_splitk", "xl_prefill_kv_split")

    def __init__(self, real):
        self._real = real
        self._wrapped = {}
        self.records = []        # (name, start_event, stop_event)
        self.enabled = True

    def __getattr__(self, name):
        f = getattr(self._real, name)
        if name in self._PLAIN or not name.startswith("xl_"):
            return f
        w = self._wrapped.get(name)
        if w is None:
            def w(*a, _f=f, _n=name):
                if not self.enabled or torch.cuda.is_current_stream_capturing():
                    return _f(*a)
                e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
                e0.record()
                rc = _f(*a)
                e1.record()
                self.records.append((_n, e0, e1))
                return rc
            self._wrapped[name] = w
        return w

    def reset(self):
        self.records = []

    def summary(self):
        """{entry point: (launches, total device ms)} since the last reset (synchronises the device)."""
        torch.cuda.synchronize()
        out = {}
        for n, e0, e1 in self.records:
            c, t = out.get(n, (0, 0.0))
            out[n] = (c + 1, t + e0.elapsed_time(e1))
        return out


def lib():
    global _lib
    if _lib is None:
        if not os.path.exists(_LIB_PATH):
            raise RuntimeError(f"{_LIB_PATH} is missing: run `python -m xllm_wxh_b200.build_ext` (needs nvcc)")
        real = ctypes.CDLL(_LIB_PATH)
        real.xl_read_status.restype = c_int
        real.xl_sm_count.restype = c_int
        _lib = _TimedLib(real) if os.environ.get("XLLM_KERNEL_TIMING") == "1" else real
    return _lib


def kernel_timing():
    """The `_TimedLib` when kernel timing is on, else None."""
    L = lib()
    return L if isinstance(L, _TimedLib) else None


def _ptr(t: Optional[torch.Tensor]):
    return c_void_p(t.data_ptr()) if t is not None else c_void_p(0)


def _stream():
    return c_void_p(torch.cuda.current_stream().cuda_stream)


def _check(rc: int, name: str):
    if rc != 0:
        raise RuntimeError(f"{name} failed with code {rc} (-2: unsupported shape/alignment, -1: launch error)")


def read_status() -> int:
    """Device status word: non-zero when a bounded wait inside a kernel gave up (synchronises the device)."""
    return int(lib().xl_read_status())


def sm_count() -> int:
    return int(lib().xl_sm_count())


# ----------------------------------------------------------------------------- GEMM
def _tc_gemm_ok(x: torch.Tensor, w: torch.Tensor, n_align: int = 8) -> bool:
    """Whether the tensor-core GEMMs serve x [M, K] and w [..., N, K]: bf16, rows on 16-byte boundaries, N a multiple of
    `n_align`."""
    return (x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and w.shape[-1] % 8 == 0 and w.shape[-2] % n_align == 0 and
            x.stride(0) % 8 == 0 and (x.data_ptr() | w.data_ptr()) % 16 == 0)


def _gemm_simt(x2: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype, bias: Optional[torch.Tensor] = None, act: int = 0,
               cap: float = 0.0) -> torch.Tensor:
    """The fp32-pipe GEMM: fp32 operands, or bf16 ones of any shape; act(x w^T + bias)."""
    global launch_count
    assert x2.dtype == w.dtype and x2.dtype in (torch.float32, torch.bfloat16) and w.stride(-1) == 1
    assert bias is None or bias.dtype == w.dtype
    M, K = x2.shape
    N = w.shape[0]
    out = torch.empty((M, N), dtype=out_dtype, device=x2.device)
    if M > 0:
        _check(lib().xl_gemm_simt(_ptr(x2), _ptr(w), _ptr(out), _ptr(bias), c_int(act), c_float(cap), c_int(M), c_int(N), c_int(K), c_long(x2.stride(0)),
                                  c_long(w.stride(0)), c_long(N), c_int(int(x2.dtype == torch.float32)), c_int(int(out_dtype == torch.float32)), _stream()),
               "xl_gemm_simt")
        launch_count += 1
    return out


def linear_f32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x w^T with the fp32 sums kept (router logits); x and w bf16 or fp32."""
    global launch_count
    if x.stride(-1) != 1:
        x = x.contiguous()
    M, K = x.shape
    N = w.shape[0]
    if not _tc_gemm_ok(x, w, 1):
        return _gemm_simt(x, w, torch.float32)
    out = torch.empty((M, N), dtype=torch.float32, device=x.device)
    if M > 0:
        _check(lib().xl_gemm_bf16_f32(_ptr(x), _ptr(w), _ptr(out), c_int(M), c_int(N), c_int(K), c_int(x.stride(0)), c_int(w.stride(0)),
                                      c_int(N), _stream()), "xl_gemm_bf16_f32")
        launch_count += 1
    return out


def linear(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    global launch_count
    if x.dtype == torch.float32 or (out is None and not _tc_gemm_ok(x.reshape(-1, x.shape[-1]), w)):
        assert out is None
        x2 = x.reshape(-1, x.shape[-1])
        return _gemm_simt(x2 if x2.stride(-1) == 1 else x2.contiguous(), w, x.dtype, bias).reshape(x.shape[:-1] + (w.shape[0],))
    assert x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16, "GEMM kernel is bf16"
    x2 = x.reshape(-1, x.shape[-1])
    if x2.stride(-1) != 1:
        x2 = x2.contiguous()
    M, K = x2.shape
    N = w.shape[0]
    assert w.shape[1] == K and w.stride(-1) == 1
    if out is None:
        out = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
    if M > 0:
        rc = lib().xl_gemm_bf16(_ptr(x2), _ptr(w), _ptr(out), _ptr(bias), c_int(M), c_int(N), c_int(K), c_int(x2.stride(0)),
                                c_int(w.stride(0)), c_int(out.stride(0)), _stream())
        _check(rc, "xl_gemm_bf16")
        launch_count += 1
    return out.reshape(x.shape[:-1] + (N,))


PLAIN_ACTS = {"relu2": 1, "tanh": 2, "softcap": 3}


def act_linear(x: torch.Tensor, w: torch.Tensor, act: str, cap: float = 0.0) -> torch.Tensor:
    """act(x w^T), applied to the fp32 sums in the GEMM epilogue."""
    global launch_count
    if x.stride(-1) != 1:
        x = x.contiguous()
    if not _tc_gemm_ok(x, w):
        return _gemm_simt(x, w, x.dtype, None, PLAIN_ACTS[act], cap)
    M, K = x.shape
    N = w.shape[0]
    out = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
    if M > 0:
        _check(lib().xl_gemm_bf16_act(_ptr(x), _ptr(w), _ptr(out), c_int(M), c_int(N), c_int(K), c_int(x.stride(0)), c_int(w.stride(0)),
                                      c_int(N), c_int(PLAIN_ACTS[act]), c_float(cap), _stream()), "xl_gemm_bf16_act")
        launch_count += 1
    return out


def linear_softcap(x: torch.Tensor, w: torch.Tensor, cap: float) -> torch.Tensor:
    return act_linear(x, w, "softcap", cap)


ACTS = {"silu": 0, "gelu_tanh": 1, "clamped": 2}


def linear_gated(x: torch.Tensor, w_interleaved: torch.Tensor, act: str, limit: float = 0.0) -> torch.Tensor:
    """gate_up GEMM whose epilogue applies act(gate) * up; `w_interleaved` from `interleave_gate_up`."""
    global launch_count
    if x.stride(-1) != 1:
        x = x.contiguous()
    M, K = x.shape
    N = w_interleaved.shape[0]
    out = torch.empty((M, N // 2), dtype=torch.bfloat16, device=x.device)
    if M > 0:
        _check(lib().xl_gemm_bf16_gated(_ptr(x), _ptr(w_interleaved), _ptr(out), c_int(M), c_int(N), c_int(K), c_int(x.stride(0)),
                                        c_int(w_interleaved.stride(0)), c_int(out.stride(0)), c_int(ACTS[act]), c_float(limit),
                                        _stream()), "xl_gemm_bf16_gated")
        launch_count += 1
    return out


def gated_act(x: torch.Tensor, act: str, limit: float = 0.0) -> torch.Tensor:
    """[T, 2I] = [gate | up] -> act(gate) * up (bf16 or fp32, any I)."""
    global launch_count
    T, I2 = x.shape
    assert x.is_contiguous()
    out = torch.empty((T, I2 // 2), dtype=x.dtype, device=x.device)
    _check(lib().xl_gated_act(_ptr(x), _ptr(out), c_int(T), c_int(I2 // 2), c_int(ACTS[act]), c_float(limit),
                              c_int(int(x.dtype == torch.float32)), _stream()), "xl_gated_act")
    launch_count += 1
    return out


def linear_swiglu(x: torch.Tensor, w_interleaved: torch.Tensor) -> torch.Tensor:
    """gate_up GEMM with the SwiGLU epilogue; `w_interleaved` from `interleave_gate_up`."""
    global launch_count
    if x.stride(-1) != 1:
        x = x.contiguous()
    M, K = x.shape
    N = w_interleaved.shape[0]
    out = torch.empty((M, N // 2), dtype=torch.bfloat16, device=x.device)
    if M > 0:
        rc = lib().xl_gemm_bf16_swiglu(_ptr(x), _ptr(w_interleaved), _ptr(out), c_int(M), c_int(N), c_int(K), c_int(x.stride(0)),
                                       c_int(w_interleaved.stride(0)), c_int(out.stride(0)), _stream())
        _check(rc, "xl_gemm_bf16_swiglu")
        launch_count += 1
    return out


def interleave_gate_up(w: torch.Tensor) -> torch.Tensor:
    """[2I, K] (gate rows then up rows) -> rows interleaved in groups of 16 (16 gate, 16 up, ...)."""
    I = w.shape[0] // 2
    assert I % 16 == 0
    g, u = w[:I].reshape(I // 16, 16, -1), w[I:].reshape(I // 16, 16, -1)
    return torch.stack([g, u], dim=1).reshape(2 * I, -1).contiguous()


def gemm_force_bn(bn: int):
    lib().xl_gemm_force_bn(c_int(bn))


def gemm_set_mode(mode: int):
    """0: choose per problem; 1: single-CTA tiles only; 2: CTA-pair (`cta_group::2`) tiles whenever M > 128."""
    lib().xl_gemm_set_mode(c_int(mode))


# ----------------------------------------------------------------------------- elementwise
def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    global launch_count
    shp = x.shape
    x2 = x.reshape(-1, shp[-1])
    if x2.stride(-1) != 1:
        x2 = x2.contiguous()
    out = torch.empty((x2.shape[0], shp[-1]), dtype=x.dtype, device=x.device)
    _check(lib().xl_rms_norm(_ptr(x2), _ptr(w), _ptr(out), c_int(x2.shape[0]), c_int(shp[-1]), c_int(x2.stride(0)), c_float(eps),
                             _stream()), "xl_rms_norm")
    launch_count += 1
    return out.reshape(shp)


def add_rms_norm(x: torch.Tensor, residual: torch.Tensor, w: torch.Tensor, eps: float) -> Tuple[torch.Tensor, torch.Tensor]:
    global launch_count
    T, H = x.shape
    assert residual.is_contiguous()
    if x.stride(-1) != 1:
        x = x.contiguous()
    out = torch.empty((T, H), dtype=x.dtype, device=x.device)
    res_out = torch.empty((T, H), dtype=x.dtype, device=x.device)
    _check(lib().xl_add_rms_norm(_ptr(x), _ptr(residual), _ptr(w), _ptr(out), _ptr(res_out), c_int(T), c_int(H),
                                 c_int(x.stride(0)), c_float(eps), _stream()), "xl_add_rms_norm")
    launch_count += 1
    return out, res_out


def silu_and_mul(x: torch.Tensor) -> torch.Tensor:
    global launch_count
    T, I2 = x.shape
    out = torch.empty((T, I2 // 2), dtype=x.dtype, device=x.device)
    _check(lib().xl_silu_mul(_ptr(x), _ptr(out), c_int(T), c_int(I2 // 2), c_int(x.stride(0)), _stream()), "xl_silu_mul")
    launch_count += 1
    return out


def embedding(ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    global launch_count
    T = ids.numel()
    V, H = table.shape
    out = torch.empty((T, H), dtype=table.dtype, device=table.device)
    _check(lib().xl_embedding(_ptr(ids), _ptr(table), _ptr(out), c_int(T), c_int(H), c_int(V), _stream()), "xl_embedding")
    launch_count += 1
    return out


def rope_qknorm_kvwrite(qkv, positions, slots, cos_sin, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, head_dim):
    global launch_count
    T = qkv.shape[0]
    assert qkv.is_contiguous() and cos_sin.dtype == torch.float32 and cos_sin.shape[-1] == head_dim
    cache_slots = k_cache.shape[0] * k_cache.shape[1]
    _check(lib().xl_rope_qknorm_kvwrite(_ptr(qkv), _ptr(positions), _ptr(slots), _ptr(cos_sin), _ptr(q_w), _ptr(k_w),
                                        _ptr(k_cache), _ptr(v_cache), c_int(T), c_int(n_q), c_int(n_kv), c_int(head_dim),
                                        c_float(eps), c_long(cache_slots), _stream()), "xl_rope_qknorm_kvwrite")
    launch_count += 1
    return qkv[:, :n_q * head_dim]


# ----------------------------------------------------------------------------- norms before and after a sublayer, fp32 residual
def _f32flag(t: torch.Tensor):
    assert t.dtype in (torch.float32, torch.bfloat16)
    return c_int(int(t.dtype == torch.float32))


def _embed_norm(ids, table, scale, positions, pos_table, x, keep_x, w_next, eps, w_offset, w_rows=None) -> torch.Tensor:
    global launch_count
    T, H = x.shape
    assert x.is_contiguous() and x.dtype == torch.float32 and ids.numel() == T and table.shape[1] == H and w_next.dtype == table.dtype
    assert pos_table is None or (pos_table.dtype == table.dtype and pos_table.is_contiguous() and pos_table.shape[1] == H)
    h = torch.empty((T, H), dtype=table.dtype, device=table.device)
    _check(lib().xl_embed_rms_norm(_ptr(ids), _ptr(table), c_float(scale), _ptr(positions), _ptr(pos_table),
                                   c_int(0 if pos_table is None else pos_table.shape[0]), _ptr(w_rows), c_int(int(keep_x)), _ptr(x), _ptr(w_next),
                                   c_float(w_offset), _ptr(h), c_int(T), c_int(H), c_int(table.shape[0]), c_float(eps), _f32flag(table),
                                   _stream()), "xl_embed_rms_norm")
    launch_count += 1
    return h


def embed_rms_norm(ids: torch.Tensor, table: torch.Tensor, scale: float, w_next: torch.Tensor, eps: float, positions=None, pos_table=None,
                   w_offset: float = 0.0, w_rows: Optional[torch.Tensor] = None):
    """(fp32 residual x = table[ids] * scale (+ pos_table[positions]), or rms of that times w_rows, rms(x) * (w_next + w_offset))."""
    assert w_rows is None or (w_rows.dtype == table.dtype and w_rows.numel() == table.shape[1])
    x = torch.empty((ids.numel(), table.shape[1]), dtype=torch.float32, device=table.device)
    return x, _embed_norm(ids, table, scale, positions, pos_table, x, False, w_next, eps, w_offset, w_rows)


def lead_norm(lead, x: torch.Tensor, w_next: torch.Tensor, eps: float, w_offset: float = 0.0) -> torch.Tensor:
    """x += embedding rows; returns rms(x) * (w_next + w_offset)."""
    return _embed_norm(*lead, x, True, w_next, eps, w_offset)


def _lead_args(lead, H: int, dtype: torch.dtype):
    if lead is None:
        return c_void_p(0), c_void_p(0), c_int(0), c_float(0.0), c_void_p(0), c_void_p(0), c_int(0)
    ids, table, scale, positions, pos = lead
    for t in (table, pos):
        assert t is None or (t.dtype == dtype and t.is_contiguous() and t.shape[1] == H)
    return (_ptr(ids), _ptr(table), c_int(table.shape[0]), c_float(scale), _ptr(positions), _ptr(pos), c_int(0 if pos is None else pos.shape[0]))


def post_norm_add_norm(y: torch.Tensor, x: torch.Tensor, w_post: torch.Tensor, w_next: torch.Tensor, eps: float) -> torch.Tensor:
    """x += rms(y) * w_post in place; returns rms(x) * w_next."""
    global launch_count
    T, H = y.shape
    assert y.is_contiguous() and x.is_contiguous() and x.dtype == torch.float32
    h = torch.empty_like(y)
    _check(lib().xl_post_norm_add_norm(_ptr(y), _ptr(x), _ptr(w_post), _ptr(w_next), _ptr(h), c_int(T), c_int(H), c_float(eps),
                                       _f32flag(y), _stream()), "xl_post_norm_add_norm")
    launch_count += 1
    return h


def branches_post_norm_add_norm(ya, yb, w_a, w_b, scale, x, w_post, w_next, eps) -> torch.Tensor:
    """y = scale * (rms(ya) * w_a + rms(yb) * w_b); x += rms(y) * w_post in place; returns rms(x) * w_next."""
    global launch_count
    T, H = ya.shape
    assert ya.is_contiguous() and yb.is_contiguous() and ya.shape == yb.shape == x.shape and x.is_contiguous() and x.dtype == torch.float32
    h = torch.empty_like(ya)
    _check(lib().xl_branches_post_norm_add_norm(_ptr(ya), _ptr(yb), _ptr(w_a), _ptr(w_b), c_float(scale), _ptr(x), _ptr(w_post), _ptr(w_next),
                                                _ptr(h), c_int(T), c_int(H), c_float(eps), _f32flag(ya), _stream()),
           "xl_branches_post_norm_add_norm")
    launch_count += 1
    return h


def _rot_args(rot):
    """(table, positions, dims, rows, interleaved) of a rotation (table of `reference.rotary_table`, positions, interleaved)."""
    if rot is None:
        return c_void_p(0), c_void_p(0), c_int(0), c_int(0), c_int(0)
    table, positions, interleaved = rot
    assert table.dtype == torch.float32 and table.is_contiguous()
    return _ptr(table), _ptr(positions), c_int(table.shape[1]), c_int(table.shape[0]), c_int(int(interleaved))


def qknorm_kvwrite(qkv, slots, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, rot=None):
    """Per-head RMSNorm of q (in place) and k, the rotation `rot` behind it, k and v into the paged caches; returns q
    [T, n_q * dk] (a view of qkv)."""
    global launch_count
    T = qkv.shape[0]
    dk, n_v, dv = k_cache.shape[-1], v_cache.shape[-2], v_cache.shape[-1]
    assert qkv.is_contiguous() and qkv.shape[1] == (n_q + n_kv) * dk + n_v * dv and k_cache.dtype == qkv.dtype
    _check(lib().xl_qknorm_kvwrite(_ptr(qkv), _ptr(slots), _ptr(q_w), _ptr(k_w), _ptr(k_cache), _ptr(v_cache), c_int(T), c_int(n_q),
                                   c_int(n_kv), c_int(n_v), c_int(dk), c_int(dv), c_float(eps), c_long(k_cache.shape[0] * k_cache.shape[1]),
                                   *_rot_args(rot), _f32flag(qkv), _stream()), "xl_qknorm_kvwrite")
    launch_count += 1
    return qkv[:, :n_q * dk]


# ----------------------------------------------------------------------------- norms before a sublayer only, fp32 residual
def add_norm(y: torch.Tensor, x: torch.Tensor, mult: float, w_next: torch.Tensor, eps: float, vec: Optional[torch.Tensor] = None,
             w_offset: float = 0.0, lead=None) -> torch.Tensor:
    """x += mult * y, or vec * y, + the embedding rows of `lead`, in place; returns rms(x) * (w_next + w_offset)."""
    global launch_count
    T, H = y.shape
    assert y.is_contiguous() and x.is_contiguous() and x.dtype == torch.float32 and (vec is None or vec.dtype == y.dtype)
    h = torch.empty_like(y)
    _check(lib().xl_add_norm(_ptr(y), _ptr(x), c_float(mult), _ptr(vec), _ptr(w_next), c_float(w_offset), _ptr(h), c_int(T), c_int(H),
                             c_float(eps), *_lead_args(lead, H, y.dtype), _f32flag(y), _stream()), "xl_add_norm")
    launch_count += 1
    return h


def replace_norm(y: torch.Tensor, vec: torch.Tensor, x: torch.Tensor, w_next: torch.Tensor, eps: float) -> torch.Tensor:
    """x = y + vec (y, vec, x fp32); returns rms(x) * w_next."""
    global launch_count
    T, H = y.shape
    assert y.is_contiguous() and x.is_contiguous() and y.dtype == x.dtype == vec.dtype == torch.float32
    h = torch.empty((T, H), dtype=w_next.dtype, device=y.device)
    _check(lib().xl_replace_norm(_ptr(y), _ptr(vec), _ptr(x), _ptr(w_next), _ptr(h), c_int(T), c_int(H), c_float(eps), _f32flag(h),
                                 _stream()), "xl_replace_norm")
    launch_count += 1
    return h


def split_rows(x: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, scale: float) -> torch.Tensor:
    global launch_count
    T, W = x.shape
    assert x.is_contiguous() and table.is_contiguous() and x.dtype == torch.float32
    out = torch.empty((T, (2 if table.dtype == torch.float32 else 3) * W), dtype=table.dtype, device=x.device)
    _check(lib().xl_split_rows(_ptr(x), _ptr(ids), _ptr(table), c_float(scale), _ptr(out), c_int(T), c_int(W), c_int(table.shape[0]),
                               _f32flag(table), _stream()), "xl_split_rows")
    launch_count += 1
    return out


def qknorm_all_kvwrite(qkv, slots, q_w, k_w, eps, k_cache, v_cache, n_q, n_kv, rot=None, mix=None):
    """RMSNorm over all query and over all key columns, the rotation `rot` behind it, k and v into the paged caches; rows of qkv may
    hold more behind v.  Returns q [T, n_q * dk] (a view of qkv), or with `mix` the queries [T, n_q * n_kv * dk] of mixed scores."""
    global launch_count
    T = qkv.shape[0]
    dk, dv = k_cache.shape[-1], v_cache.shape[-1]
    assert qkv.stride(1) == 1 and qkv.shape[1] >= (n_q + n_kv) * dk + n_kv * dv and k_cache.dtype == qkv.dtype
    wide = None
    if mix is not None:
        assert mix.dtype == torch.float32 and mix.is_contiguous() and mix.shape == (n_q, n_q)
        wide = torch.empty((T, n_q * n_kv * dk), dtype=qkv.dtype, device=qkv.device)
    _check(lib().xl_qknorm_all_kvwrite(_ptr(qkv), _ptr(slots), _ptr(q_w), _ptr(k_w), _ptr(k_cache), _ptr(v_cache), c_int(T), c_int(n_q),
                                       c_int(n_kv), c_int(dk), c_int(n_kv * dv), c_long(qkv.stride(0)), c_float(eps),
                                       c_long(k_cache.shape[0] * k_cache.shape[1]), *_rot_args(rot), _ptr(mix), _ptr(wide), _f32flag(qkv),
                                       _stream()), "xl_qknorm_all_kvwrite")
    launch_count += 1
    return qkv[:, :n_q * dk] if wide is None else wide


def gate_into(o: torch.Tensor, gate: torch.Tensor, scale: float, out: torch.Tensor) -> None:
    global launch_count
    T, n = o.shape
    assert o.is_contiguous() and gate.shape == out.shape == o.shape and gate.stride(1) == out.stride(1) == 1
    _check(lib().xl_sigmoid_gate(_ptr(o), _ptr(gate), _ptr(out), c_int(T), c_int(n), c_long(gate.stride(0)), c_long(out.stride(0)),
                                 c_float(scale), _f32flag(o), _stream()), "xl_sigmoid_gate")
    launch_count += 1


# ----------------------------------------------------------------------------- latent attention of any size
def latent_down(low, q_rank, kv_rank, q_w, kv_w, eps, rot, slots, cache):
    global launch_count
    T = low.shape[0]
    assert low.stride(1) == 1 and low.shape[1] == q_rank + cache.shape[-1] and cache.dtype == low.dtype
    assert cache.shape[-1] == kv_rank + rot[0].shape[1]
    c_q = torch.empty((T, q_rank), dtype=low.dtype, device=low.device)
    _check(lib().xl_latent_down(_ptr(low), _ptr(q_w), _ptr(kv_w), _ptr(c_q), _ptr(cache), _ptr(slots), c_int(T), c_int(q_rank), c_int(kv_rank),
                                c_long(low.stride(0)), c_float(eps), c_long(cache.shape[0] * cache.shape[1]), *_rot_args(rot), _f32flag(low),
                                _stream()), "xl_latent_down")
    launch_count += 1
    return c_q


def rotate_into(x, rot, out) -> None:
    global launch_count
    T, H, d = x.shape
    assert out.shape == x.shape and d == rot[0].shape[1] and x.stride(2) == out.stride(2) == 1 and x.dtype == out.dtype
    _check(lib().xl_rotate(_ptr(x), _ptr(out), c_int(T), c_int(H), c_long(x.stride(0)), c_long(x.stride(1)), c_long(out.stride(0)),
                           c_long(out.stride(1)), *_rot_args(rot), _f32flag(x), _stream()), "xl_rotate")
    launch_count += 1


def _head_layout(t: torch.Tensor):
    """(pitch, rows from one head to the next, columns from one head to the next) of a view [H, T, n], or None."""
    H, T, n = t.shape
    if t.stride(2) != 1:
        return None
    if t.stride(0) == T * t.stride(1) and t.stride(1) >= n:
        return t.stride(1), T, 0                      # head-major
    return (t.stride(1), 0, t.stride(0)) if t.stride(1) >= (H - 1) * t.stride(0) + n else None


def heads_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out[h] = x[h] w[h]^T: x [H, T, K], w [H, N, K], out [H, T, N]; x and out may be views of token-major tensors."""
    global launch_count
    H, T, K = x.shape
    N = w.shape[1]
    assert w.shape == (H, N, K) and w.is_contiguous() and out.shape == (H, T, N) and x.dtype == w.dtype == out.dtype
    assert x.stride(2) == out.stride(2) == 1
    if T == 0:
        return out
    a, c = _head_layout(x), _head_layout(out)
    if (x.dtype == torch.bfloat16 and a and c and K % 8 == 0 and N % 8 == 0 and a[0] % 8 == 0 and a[2] % 8 == 0 and c[0] % 8 == 0 and
            c[2] % 8 == 0 and (x.data_ptr() | w.data_ptr() | out.data_ptr()) % 16 == 0):
        _check(lib().xl_gemm_bf16_heads(_ptr(x), _ptr(w), _ptr(out), c_int(T), c_int(N), c_int(K), c_int(a[0]), c_int(c[0]), c_int(H),
                                        c_int(a[1]), c_int(a[2]), c_int(c[1]), c_int(c[2]), _stream()), "xl_gemm_bf16_heads")
    else:
        _check(lib().xl_gemm_simt_batched(_ptr(x), _ptr(w), _ptr(out), c_int(H), c_int(T), c_int(N), c_int(K), c_long(x.stride(1)), c_long(K),
                                          c_long(out.stride(1)), c_long(x.stride(0)), c_long(N * K), c_long(out.stride(0)), _f32flag(x),
                                          _stream()), "xl_gemm_simt_batched")
    launch_count += 1
    return out


def mla_serves(heads: int, kv_rank: int, rot_dim: int, dtype: torch.dtype) -> bool:
    """Whether the kernels of `mla_attention` serve a latent attention of these sizes."""
    return dtype == torch.bfloat16 and kv_rank == 512 and rot_dim == 64 and ((heads <= 128 and 128 % heads == 0) or heads % 16 == 0)


def latent_attention_mla(q, w_uk, w_uv, cache, inp, rot, scale, dim):
    """`ops.latent_attention` through the head-major kernels of `mla_attention`."""
    T, H, _ = q.shape
    C = w_uk.shape[1]
    lat = torch.empty((H, T, C), dtype=q.dtype, device=q.device)
    heads_linear(q[..., :dim].transpose(0, 1), w_uk, lat)
    q_rot = torch.empty((H, T, q.shape[2] - dim), dtype=q.dtype, device=q.device)
    rotate_into(q[..., dim:], rot, q_rot.transpose(0, 1))
    o = mla_attention(lat, q_rot, cache, inp, scale, C)
    out = torch.empty((T, H, w_uv.shape[1]), dtype=q.dtype, device=q.device)
    heads_linear(o, w_uv, out.transpose(0, 1))
    return out.flatten(1)


# ----------------------------------------------------------------------------- recurrent layers
def _state_args(inp, state):
    assert state.is_contiguous()
    n = inp.B if inp.padded else inp.n_seqs
    return n, (_ptr(inp.q_cu), _ptr(inp.kv_lens), _ptr(inp.state_slots), c_int(n), c_int(state.shape[0]))


def _rows_out(inp, shape, like):
    """Rows that belong to no sequence (padding) are written by no recurrent kernel: keep them finite."""
    return (torch.zeros if inp.padded else torch.empty)(shape, dtype=like.dtype, device=like.device)


def token_shift(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor, inp) -> torch.Tensor:
    """[n, T, W]: h + (predecessor - h) * mu[i]; the record of every sequence in `last` [slots, W] becomes its last row."""
    global launch_count
    T, W = h.shape
    assert h.is_contiguous() and mu.is_contiguous() and mu.dtype == last.dtype == h.dtype
    n, seqs = _state_args(inp, last)
    out = torch.empty((mu.shape[0], T, W), dtype=h.dtype, device=h.device)
    _check(lib().xl_token_shift(_ptr(h), _ptr(mu), _ptr(last), _ptr(out), _ptr(inp.token_seq), *seqs, c_int(T), c_int(W),
                                c_int(mu.shape[0]), _f32flag(h), _stream()), "xl_token_shift")
    launch_count += 1
    return out


def causal_conv(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor], state: torch.Tensor, inp, act: str = "none",
                residual: bool = False) -> torch.Tensor:
    """act(b + causal convolution of x [T, C] (may be a strided view) with w [taps, C]) (+ x); act "silu" or "none"; state
    [slots, taps - 1, C]."""
    global launch_count
    T, C = x.shape
    assert x.stride(1) == 1 and w.is_contiguous() and w.dtype == state.dtype == x.dtype and (b is None or b.dtype == x.dtype)
    n, seqs = _state_args(inp, state)
    out = _rows_out(inp, (T, C), x)
    _check(lib().xl_causal_conv(_ptr(x), _ptr(w), _ptr(b), _ptr(state), _ptr(out), _ptr(inp.token_seq), *seqs, c_int(T), c_int(C),
                                c_int(w.shape[0]), c_long(x.stride(0)), c_int(int(inp.has_prefill)), c_int(int(act == "silu")),
                                c_int(int(residual)), _f32flag(x), _stream()), "xl_causal_conv")
    launch_count += 2 if inp.has_prefill and w.shape[0] > 1 else 1
    return out


mix_force_rows = 0        # > 0: that many rows per segment of time_mix (tests)


def mix_segment_rows(T: int, H: int, d: int) -> int:
    """Rows per segment of the time mixing of longer portions: short enough that segments x heads fill the device a few times
    over, long enough that the states between segments stay small beside the rows' own work."""
    if mix_force_rows > 0:
        return mix_force_rows
    want = 8 * sm_count() * 64 // max(64, d)
    L = max(1, T * H // want)
    return min(512, max(64, 1 << (L.bit_length() - 1)))


def _segments(inp, T: int, n: int, H: int, dk: int, dv: int, record: int, device):
    """(segment arguments of a matrix-state kernel, whether longer portions may occur, launches): rows per segment, how many there
    can be and the workspace of the states between them."""
    has_long = bool(inp.has_prefill) and T > 1
    if not has_long:
        return (c_int(2), c_int(0), c_void_p(0), c_void_p(0)), (), False, 1
    L = mix_segment_rows(T, H, max(dk, dv))
    cap = T // L + min(n, T // 2)                           # every portion of two and more rows ends with one partly filled segment
    ws = wp = None
    if (T if inp.padded else inp.max_q) > L and max(dk, dv) <= 128:
        ws = torch.empty((cap, H, record), dtype=torch.float32, device=device)
        wp = torch.empty((cap, H, dk), dtype=torch.float32, device=device)
    return (c_int(L), c_int(cap), _ptr(ws), _ptr(wp)), (ws, wp), True, 2 if ws is None else 4


def _check_rows(r, k, v, gate, out, T, dk, dv):
    for t, width in ((r, dk), (k, dk), (v, dv)):
        assert t.stride(1) == 1 and t.stride(0) == r.stride(0) and t.dtype == out.dtype and t.shape == (T, width)
    assert gate.stride(1) == out.stride(1) == 1 and gate.shape == (T, dv)


def time_mix(r, k, v, z, w0, u, gate, norm_w, scale, eps, state, inp, out) -> None:
    global launch_count
    H, d = u.shape
    T = r.shape[0]
    _check_rows(r, k, v, gate, out, T, H * d, H * d)
    assert z.is_contiguous() and z.dtype == w0.dtype == u.dtype == state.dtype == torch.float32
    n, seqs = _state_args(inp, state)
    if inp.padded:
        out.zero_()
    seg, keep, has_long, launches = _segments(inp, T, n, H, d, d, d * d, r.device)
    _check(lib().xl_time_mix(_ptr(r), _ptr(k), _ptr(v), _ptr(z), _ptr(w0), _ptr(u), _ptr(gate), _ptr(norm_w), c_float(scale), c_float(eps),
                             _ptr(state), _ptr(out), *seqs, c_int(H), c_int(d), c_long(r.stride(0)), c_long(gate.stride(0)),
                             c_long(out.stride(0)), *seg, c_int(int(has_long)), c_int(1), _f32flag(r), _stream()), "xl_time_mix")
    launch_count += launches


def gated_memory(q, k, v, z, bias, inv_tau, gate, norm_w, eps, state, inp) -> torch.Tensor:
    global launch_count
    _, H, dk, dv = state.shape
    T = q.shape[0]
    n, seqs = _state_args(inp, state)
    out = _rows_out(inp, (T, H * dv), q)
    _check_rows(q, k, v, gate, out, T, H * dk, H * dv)
    assert z.is_contiguous() and z.shape == (T, H * dk) and bias.numel() == H * dk and norm_w.numel() == dv
    assert z.dtype == bias.dtype == state.dtype == torch.float32 and norm_w.dtype == q.dtype
    seg, keep, has_long, launches = _segments(inp, T, n, H, dk, dv, dk * dv, q.device)
    _check(lib().xl_gated_memory(_ptr(q), _ptr(k), _ptr(v), _ptr(z), _ptr(bias), c_float(inv_tau), _ptr(gate), _ptr(norm_w), c_float(eps),
                                 _ptr(state), _ptr(out), *seqs, c_int(H), c_int(dk), c_int(dv), c_long(q.stride(0)), c_long(gate.stride(0)),
                                 c_long(out.stride(0)), *seg, c_int(int(has_long)), c_int(1), _f32flag(q), _stream()), "xl_gated_memory")
    launch_count += launches
    return out


def matrix_memory(q, k, v, gates, bias, cap, gate, norm_w, eps, state, top, inp) -> torch.Tensor:
    global launch_count
    H = top.shape[1]
    T, dk, dv = q.shape[0], q.shape[1] // H, v.shape[1] // H
    n, seqs = _state_args(inp, state)
    out = _rows_out(inp, (T, H * dv), q)
    _check_rows(q, k, v, gate, out, T, H * dk, H * dv)
    assert gates.is_contiguous() and gates.shape == (T, 2 * H) and bias.numel() == 2 * H and norm_w.numel() == H * dv
    assert state.shape == (state.shape[0], H, dk * dv + dk) and top.shape[0] == state.shape[0] and top.is_contiguous()
    assert gates.dtype == bias.dtype == state.dtype == top.dtype == torch.float32 and norm_w.dtype == q.dtype
    seg, keep, has_long, launches = _segments(inp, T, n, H, dk, dv, dk * dv + dk, q.device)
    fi = torch.empty((3, H, T), dtype=torch.float32, device=q.device)
    _check(lib().xl_matrix_memory(_ptr(q), _ptr(k), _ptr(v), _ptr(gates), _ptr(bias), c_float(cap), _ptr(gate), _ptr(norm_w), c_float(eps),
                                  _ptr(state), _ptr(top), _ptr(out), *seqs, c_int(H), c_int(dk), c_int(dv), c_long(q.stride(0)),
                                  c_long(gate.stride(0)), c_long(out.stride(0)), *seg, _ptr(fi), c_int(T), c_int(int(has_long)), c_int(1),
                                  _f32flag(q), _stream()), "xl_matrix_memory")
    launch_count += launches + int(has_long)
    return out


def selective_scan(x, dt, dt_bias, A, B, C, D, z, state, inp) -> torch.Tensor:
    global launch_count
    T, ch = x.shape
    N = A.shape[1]
    assert x.is_contiguous() and dt.is_contiguous() and dt.dtype == dt_bias.dtype == A.dtype == D.dtype == state.dtype == torch.float32
    assert B.stride(1) == C.stride(1) == z.stride(1) == 1 and B.stride(0) == C.stride(0) and B.dtype == z.dtype == x.dtype
    n, seqs = _state_args(inp, state)
    out = _rows_out(inp, (T, ch), x)
    _check(lib().xl_selective_scan(_ptr(x), _ptr(dt), _ptr(dt_bias), _ptr(A), _ptr(B), _ptr(C), _ptr(D), _ptr(z), _ptr(state), _ptr(out),
                                   *seqs, c_int(ch), c_int(N), c_long(B.stride(0)), c_long(z.stride(0)), c_int(int(inp.has_prefill)),
                                   c_int(1), _f32flag(x), _stream()), "xl_selective_scan")
    launch_count += 2 if inp.has_prefill else 1
    return out


# ----------------------------------------------------------------------------- attention
decode_kernel = "tma"     # "tma" | "cp_async" (the fallback kernel; selectable for tests and comparisons)


def prefill_use_tc(on: bool):
    """Prefill attention kernel choice: tcgen05 (default) or the mma.sync kernel (comparisons, tests)."""
    lib().xl_prefill_use_tc(c_int(int(on)))


def prefill_kv_split(mode: int):
    """Key-range split of the tcgen05 prefill kernel: 0 = never, 1 = automatic (default: when query tiles x heads leave
    SMs idle), 2..8 = that many splits (tests, measurements)."""
    lib().xl_prefill_kv_split(c_int(int(mode)))


def decode_splits(n_seqs: int, n_kv: int, max_kv: int) -> int:
    """Key-range splits of the decode kernel: fill the two CTAs each SM holds, but never spill into a second, partly
    filled wave (measured at 255 sequences x 1 KV head: one split 28 us, two 35 us)."""
    ctas = max(1, n_seqs * n_kv)
    want = (2 * sm_count()) // ctas
    by_len = max(1, max_kv // 512)
    return max(1, min(want, by_len, 16))


def paged_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, inp, scale: float, window: int = -1) -> torch.Tensor:
    """q [T, Hq, D] (may be a strided view of the qkv buffer).  Decode sequences (the leading `inp.n_decode` ones) go to the
    split-KV kernel, the rest to the prefill kernel.  In a padded step (CUDA-graph capture / replay) the launches are sized
    for the capacities of the layout and the kernels read the real decode / prefill split from the device-side header."""
    global launch_count
    from ..framework.step_input import H_NUM_DECODE, H_NUM_SEQS
    T, Hq, D = q.shape
    n_kv = k_cache.shape[2]
    block_size = k_cache.shape[1]
    L = inp.layout
    padded = inp.padded
    # padded rows belong to no sequence and are written by no kernel: keep them finite
    out = (torch.zeros if padded else torch.empty)((T, Hq * D), dtype=q.dtype, device=q.device)
    n_dec = inp.B if padded else inp.n_decode
    n_all = inp.B if padded else inp.n_seqs
    has_prefill = inp.has_prefill if padded else n_all > n_dec
    hdr = getattr(inp, "header_dev", None)       # only padded steps read it (rows built on the device carry none)
    dyn_dec = c_void_p(hdr.data_ptr() + 4 * H_NUM_DECODE) if padded else c_void_p(0)
    dyn_all = c_void_p(hdr.data_ptr() + 4 * H_NUM_SEQS) if padded else c_void_p(0)
    q_stride = q.stride(0)
    common = (_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(out), _ptr(inp.q_cu), _ptr(inp.kv_lens), _ptr(inp.block_tables))
    if n_dec > 0:
        max_kv = (L.MB_cap * block_size) if padded else inp.max_kv
        splits = decode_splits(n_dec, n_kv, max_kv)
        po = pl = None
        if splits > 1:
            rows = n_dec * max(1, 16 // (Hq // n_kv)) if padded else T
            rows = max(rows, T)
            po = torch.empty((rows, Hq, splits, D), dtype=torch.float32, device=q.device)
            pl = torch.empty((rows, Hq, splits), dtype=torch.float32, device=q.device)
        rc = -3
        if decode_kernel != "cp_async":
            rc = lib().xl_decode_attention_tma_dyn(*common, c_int(0), c_int(n_dec), c_int(L.MB_cap), c_int(block_size),
                                                   c_int(k_cache.shape[0]), c_int(Hq), c_int(n_kv), c_int(D), c_int(q_stride),
                                                   c_float(scale), c_int(window), c_int(splits), _ptr(po), _ptr(pl), dyn_dec,
                                                   _stream())
            if rc == 0 and splits > 1:
                _check(lib().xl_decode_split_merge_dyn(_ptr(po), _ptr(pl), _ptr(out), _ptr(inp.q_cu), c_int(0), c_int(n_dec),
                                                       c_int(Hq), c_int(D), c_int(splits), c_long(po.shape[0]), dyn_dec,
                                                       _stream()), "xl_decode_split_merge")
        if rc == -3:        # shape not covered by the TMA kernel: per-lane cp.async kernel
            rc = lib().xl_paged_attention_dyn(*common, c_int(0), c_int(n_dec), c_int(L.MB_cap), c_int(block_size),
                                              c_int(k_cache.shape[0]), c_int(Hq), c_int(n_kv), c_int(D), c_int(q_stride),
                                              c_float(scale), c_int(window), c_int(1), c_int(0), c_int(splits), _ptr(po),
                                              _ptr(pl), c_void_p(0), dyn_dec, c_int(T), _stream())
        _check(rc, "decode attention")
        launch_count += 1 + (1 if splits > 1 else 0)
    if has_prefill:
        # q tiles of 64 rows: every sequence adds at most one partly filled tile
        tiles = (T + 63) // 64 + n_all if padded else (inp.n_prefill_tokens + 63) // 64 + (n_all - n_dec)
        lo = 0 if padded else n_dec
        _check(lib().xl_paged_attention_dyn(*common, c_int(lo), c_int(n_all), c_int(L.MB_cap), c_int(block_size),
                                            c_int(k_cache.shape[0]), c_int(Hq), c_int(n_kv), c_int(D), c_int(q_stride),
                                            c_float(scale), c_int(window), c_int(0), c_int(tiles), c_int(1), c_void_p(0),
                                            c_void_p(0), dyn_dec, dyn_all, c_int(T), _stream()), "xl_paged_attention(prefill)")
        launch_count += 1
    return out


def paged_attention_ext(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, inp, scale: float, window: int = -1, chunk: int = 0,
                        slopes: Optional[torch.Tensor] = None, sinks: Optional[torch.Tensor] = None, keep_first: int = 0,
                        softcap: float = 0.0, mix=None, bound: float = 0.0) -> torch.Tensor:
    """Paged attention with score extensions and a value dimension of its own: q [T, Hq, dk] (may be a view of the qkv
    buffer), caches [blocks, block, Hkv, dk | dv] -> [T, Hq * dv].  score = scale q.k (bounded by softcap tanh(. / softcap)) -
    slopes[h] * distance; keys of the query's own chunk of `chunk` positions only (0: all); `keep_first` first keys stay visible
    behind the window; exp(sinks[h]) joins the softmax denominator; `mix`: differential attention (see `ops`).  The values may be
    a view of the keys; one key head may serve several value heads.  bf16 tensors with head dimensions up to 256 (128 with `mix`; multiples of 8) run on the tensor-core
    kernels, anything else on the fp32-pipe kernel."""
    global launch_count
    from ..framework.step_input import H_NUM_DECODE, H_NUM_SEQS
    T, Hq, dk = q.shape
    block_size, n_kv, dv = k_cache.shape[1], v_cache.shape[2], v_cache.shape[3]
    maps = 1 if mix is None else 2
    shared_keys = maps == 1 and n_kv > 1 and k_cache.shape[2] == 1
    assert k_cache.is_contiguous() and k_cache.shape[2] == (1 if shared_keys else n_kv * maps) and v_cache.stride(3) == 1 and v_cache.stride(0) == block_size * v_cache.stride(1)
    assert v_cache.stride(2) == dv or n_kv == 1
    L, padded = inp.layout, inp.padded
    for t in (slopes, sinks):
        assert t is None or (t.dtype == torch.float32 and t.numel() == Hq and t.is_contiguous())
    out = (torch.zeros if padded else torch.empty)((T, Hq // maps * dv), dtype=q.dtype, device=q.device)
    factor, mult, eps = mix if mix is not None else (None, 0.0, 0.0)
    last = (c_long(v_cache.stride(1)), c_int(int(shared_keys)), c_int(maps), _ptr(factor), c_float(mult), c_float(eps))
    ext = (c_float(softcap), c_float(bound)) + last
    n_dec = inp.B if padded else inp.n_decode
    n_all = inp.B if padded else inp.n_seqs
    has_prefill = inp.has_prefill if padded else n_all > n_dec
    q_stride = q.stride(0)

    def simt():
        _check(lib().xl_attention_simt(_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(out), _ptr(inp.token_seq), _ptr(inp.positions),
                                       _ptr(inp.block_tables), c_int(T), c_int(n_all), c_int(L.MB_cap), c_int(block_size),
                                       c_long(k_cache.shape[0] * block_size), c_int(Hq), c_int(n_kv), c_int(dk), c_int(dv),
                                       c_long(q_stride), c_float(scale), c_int(window), c_int(chunk), c_int(keep_first), _ptr(slopes), _ptr(sinks),
                                       c_float(softcap), *last, _f32flag(q), _stream()), "xl_attention_simt")
        return out
    most = 256 if mix is None else 128
    plain = slopes is None and softcap <= 0 and chunk <= 0 and keep_first <= 0
    wide = shared_keys and dk > 128 and dv <= 128 and plain                  # kernels of their own, for keys of any width
    if q.dtype == torch.float32 or dk % 8 or dv % 8 or (dk > most and not wide) or dv > most or q.stride(1) != dk:
        launch_count += 1
        return simt()
    hdr = getattr(inp, "header_dev", None)
    dyn_dec = c_void_p(hdr.data_ptr() + 4 * H_NUM_DECODE) if padded else c_void_p(0)
    dyn_all = c_void_p(hdr.data_ptr() + 4 * H_NUM_SEQS) if padded else c_void_p(0)
    common = (_ptr(q), _ptr(k_cache), _ptr(v_cache), _ptr(out), _ptr(inp.q_cu), _ptr(inp.kv_lens), _ptr(inp.block_tables))
    shape = (c_int(L.MB_cap), c_int(block_size), c_int(k_cache.shape[0]), c_int(Hq), c_int(n_kv), c_int(dk), c_int(dv), c_int(q_stride))
    if n_dec > 0:
        max_kv = (L.MB_cap * block_size) if padded else inp.max_kv
        if chunk > 0:
            max_kv = min(max_kv, chunk)
        if window > 0:
            max_kv = min(max_kv, window + keep_first)
        max_q = max(1, inp.max_q) if inp.n_spec > 0 else 1
        splits = decode_splits(n_dec, n_kv * -(-Hq // n_kv * max_q // 16), max_kv)
        if wide:                    # one CTA of up to 32 query rows per SM
            splits = max(1, min(sm_count() // max(1, n_dec * -(-Hq * max_q // 32)), max_kv // 512, 16))
        po = pl = None
        rows = max(T, n_dec)
        if splits > 1:
            po = torch.empty((rows, Hq, splits, dv), dtype=torch.float32, device=q.device)
            pl = torch.empty((rows, Hq, splits), dtype=torch.float32, device=q.device)
        rc = lib().xl_decode_attention_ext(*common, c_int(0), c_int(n_dec), *shape, c_float(scale), c_int(window), c_int(chunk),
                                           c_int(keep_first), _ptr(slopes), _ptr(sinks), *ext, c_int(max_q), c_int(splits), _ptr(po), _ptr(pl),
                                           c_long(rows), dyn_dec, _stream())
        if rc == -3:            # a block size outside the tensor-core kernels' limits
            launch_count += 1
            return simt()
        _check(rc, "xl_decode_attention_ext")
        launch_count += 1 + (1 if splits > 1 else 0)
    if has_prefill:
        tiles = (T + 127) // 128 + n_all if padded else (inp.n_prefill_tokens + 127) // 128 + (n_all - n_dec)
        rc = lib().xl_prefill_attention_ext(*common, c_int(0 if padded else n_dec), c_int(n_all), *shape, c_int(T), c_float(scale),
                                            c_int(window), c_int(chunk), c_int(keep_first), _ptr(slopes), _ptr(sinks), *ext, c_int(tiles), dyn_dec,
                                            dyn_all, _stream())
        if rc == -3:
            launch_count += 1
            return simt()
        _check(rc, "xl_prefill_attention_ext")
        launch_count += 1
    return out


# ----------------------------------------------------------------------------- sampling
def sample(logits: torch.Tensor, inp):
    global launch_count
    S, V = logits.shape
    dt = 0 if logits.dtype == torch.float32 else 1
    assert logits.dtype in (torch.float32, torch.bfloat16) and logits.stride(-1) == 1
    if inp.any_penalty:
        _check(lib().xl_apply_penalties(_ptr(logits), c_int(dt), c_int(S), c_int(V), c_long(logits.stride(0)), _ptr(inp.pen_cu),
                                        _ptr(inp.pen_ids), _ptr(inp.pen_counts), _ptr(inp.rep_pen), _ptr(inp.freq_pen),
                                        _ptr(inp.pres_pen), _stream()), "xl_apply_penalties")
        launch_count += 1
    tokens = torch.empty(S, dtype=torch.int32, device=logits.device)
    lp = tv = ti = None
    n_top = 0
    if inp.any_logprobs:
        lp = torch.empty(S, dtype=torch.float32, device=logits.device)
        n_top = inp.max_top_logprobs
        if n_top > 0:
            tv = torch.empty((S, n_top), dtype=torch.float32, device=logits.device)
            ti = torch.empty((S, n_top), dtype=torch.int32, device=logits.device)
    _check(lib().xl_sample(_ptr(logits), c_int(dt), c_int(S), c_int(V), c_long(logits.stride(0)), _ptr(inp.temperature),
                           _ptr(inp.top_k), _ptr(inp.top_p), _ptr(inp.seed_lo), _ptr(inp.seed_hi), _ptr(tokens), _ptr(lp),
                           c_int(n_top), _ptr(tv), _ptr(ti), _stream()), "xl_sample")
    launch_count += 1
    return tokens, lp, tv, ti


def topk_candidates(logits: torch.Tensor, inp, id_offset: int, width: int):
    """Per-shard candidates of vocabulary-parallel sampling: the top_k largest logits of every row of this vocabulary
    slice (ties at the k-th included; the arg-max for greedy rows) as (values fp32 [S, width], global ids int32 [S, width],
    overflow flag int32 [1]); unused places hold -inf / -1."""
    global launch_count
    S, V = logits.shape
    dt = 0 if logits.dtype == torch.float32 else 1
    assert logits.dtype in (torch.float32, torch.bfloat16) and logits.stride(-1) == 1
    vals = torch.empty((S, width), dtype=torch.float32, device=logits.device)
    ids = torch.empty((S, width), dtype=torch.int32, device=logits.device)
    over = torch.zeros(1, dtype=torch.int32, device=logits.device)
    _check(lib().xl_topk_candidates(_ptr(logits), c_int(dt), c_int(S), c_int(V), c_long(logits.stride(0)), _ptr(inp.temperature),
                                    _ptr(inp.top_k), c_int(id_offset), c_int(width), _ptr(vals), _ptr(ids), _ptr(over), _stream()),
           "xl_topk_candidates")
    launch_count += 1
    return vals, ids, over


# ----------------------------------------------------------------------------- MoE
def moe_router(logits, top_k, scoring="softmax", renorm=True, bias=None, n_group=1, topk_group=1, route_scale=1.0, group_score=None):
    from . import moe_cuda
    return moe_cuda.moe_router(logits, top_k, scoring, renorm, bias, n_group, topk_group, route_scale, group_score=group_score)


def moe_experts(x, w13, w2, weights, ids, expert_offset=0, interleaved=False):
    from . import moe_cuda
    return moe_cuda.moe_experts(x, w13, w2, weights, ids, expert_offset, interleaved)


# ----------------------------------------------------------------------------- MLA
class _HeadTiles:
    """Tile table that treats the heads of a head-major [Hh, T, K] tensor as the groups of a grouped GEMM."""
    _cache = {}

    def __init__(self, Hh: int, T: int, device):
        per = (T + 127) // 128
        h = torch.arange(Hh, device=device, dtype=torch.int32).repeat_interleave(per)
        i = torch.arange(per, device=device, dtype=torch.int32).repeat(Hh)
        self.tile_expert = h.contiguous()
        self.tile_row0 = (h * T + i * 128).contiguous()
        self.tile_row_end = ((h + 1) * T).contiguous()
        self.max_tiles = Hh * per
        self.num_m_tiles = torch.tensor([self.max_tiles], dtype=torch.int32, device=device)

    @classmethod
    def get(cls, Hh, T, device):
        key = (Hh, T, str(device))
        t = cls._cache.get(key)
        if t is None:
            if len(cls._cache) > 256:
                cls._cache.clear()
            t = cls._cache[key] = cls(Hh, T, device)
        return t


def _w_kc_t(w_kc: torch.Tensor) -> torch.Tensor:
    """[Hh, nope, c] -> [Hh, c, nope] (the [N, K] weight layout of the absorb GEMM).  The transposed copy lives on the weight
    tensor itself, so it goes away with it: a table keyed by the data pointer would hand a later model, whose weights the
    allocator put at the same address, the previous model's copy."""
    try:
        version = w_kc._version          # changes when the weights are rewritten in place (wake-up from sleep)
    except RuntimeError:                 # a tensor made under inference mode keeps no version
        version = 0
    t = getattr(w_kc, "_xl_kc_t", None)
    if t is None or t.shape != (w_kc.shape[0], w_kc.shape[2], w_kc.shape[1]) or getattr(w_kc, "_xl_kc_version", -1) != version:
        t = w_kc.transpose(1, 2).contiguous()
        w_kc._xl_kc_t = t
        w_kc._xl_kc_version = version
    return t


def mla_prepare(q, kv_a, positions, slots, cos_sin, kv_norm_w, eps, cache, w_kc, nope, rope, kv_lora):
    """Returns head-major tensors (q_lat [Hh, T, kv_lora], q_pe [Hh, T, rope]) for `mla_attention`."""
    global launch_count
    from . import moe_cuda
    T, Hh, _ = q.shape
    q = q.contiguous()
    kv_a = kv_a.contiguous()
    q_nope = torch.empty((Hh, T, nope), dtype=q.dtype, device=q.device)
    q_pe = torch.empty((Hh, T, rope), dtype=q.dtype, device=q.device)
    slots_total = cache.shape[0] * cache.shape[1]
    _check(lib().xl_mla_prepare(_ptr(q), _ptr(kv_a), _ptr(positions), _ptr(slots), _ptr(cos_sin), _ptr(kv_norm_w), _ptr(cache),
                                _ptr(q_nope), _ptr(q_pe), c_int(T), c_int(Hh), c_int(nope), c_int(rope), c_int(kv_lora),
                                c_float(eps), c_long(slots_total), _stream()), "xl_mla_prepare")
    launch_count += 1
    tiles = _HeadTiles.get(Hh, T, q.device)
    q_lat = moe_cuda.grouped_gemm(q_nope.view(Hh * T, nope), _w_kc_t(w_kc), tiles)
    return q_lat.view(Hh, T, kv_lora), q_pe


def mla_attention(q_lat_hm, q_pe_hm, cache, inp, scale, kv_lora):
    """Head-major in and out.  The tcgen05 kernel serves head counts that divide 128 (XLLM_MLA_TC=0: the mma.sync kernel)."""
    global launch_count
    Hh, T, C = q_lat_hm.shape
    rope = q_pe_hm.shape[-1]
    # padded rows belong to no sequence and are written by no kernel: keep them finite, since the next layer writes their latents
    # into the padding block, which tiles past a sequence's end may read
    out = (torch.zeros_like if inp.padded else torch.empty_like)(q_lat_hm)
    L = inp.layout
    n_all = inp.B if inp.padded else inp.n_seqs
    common = (_ptr(inp.q_cu), _ptr(inp.kv_lens), _ptr(inp.block_tables), c_int(0), c_int(n_all), c_int(L.MB_cap),
              c_int(cache.shape[1]), c_long(cache.shape[0] * cache.shape[1]), c_int(Hh), c_int(T), c_int(C), c_int(rope), c_float(scale))
    if Hh <= 128 and 128 % Hh == 0 and os.environ.get("XLLM_MLA_TC", "1") != "0":
        tpt = 128 // Hh
        max_tiles = (T + n_all * (tpt - 1)) // tpt + 1
        rc = lib().xl_mla_attention_tc(_ptr(q_lat_hm), _ptr(q_pe_hm), _ptr(cache), _ptr(out), *common, c_int(max_tiles), _stream())
        if rc == 0:
            launch_count += 1
            return out
        if rc != -3:
            _check(rc, "xl_mla_attention_tc")
    max_tiles = T * (Hh // 16) + n_all * Hh
    _check(lib().xl_mla_attention(_ptr(q_lat_hm), _ptr(q_pe_hm), _ptr(cache), _ptr(out), *common, c_int(max_tiles), _stream()),
           "xl_mla_attention")
    launch_count += 1
    return out


def index_scores(q, w, keys, block_tables, token_seq, positions, S: int):
    """Lightning-indexer scores [T, S] (fp32; -inf at keys after the query): q [T, n_heads, 128] bf16, w [T, n_heads] fp32
    (softmax scale folded in), keys [blocks, block, 128] bf16 read through `block_tables` [B, max_blocks] of the
    sequence `token_seq[t]`, causal by `positions[t]`.  None where the kernel does not serve the shape."""
    global launch_count
    T, NH, D = q.shape
    if D != 128 or NH not in (16, 32, 64) or T > 65535 or keys.dtype != torch.bfloat16 or q.dtype != torch.bfloat16:
        return None
    q, w, block_tables = q.contiguous(), w.contiguous(), block_tables.contiguous()
    token_seq, positions = token_seq.contiguous(), positions.contiguous()
    assert w.dtype == torch.float32 and block_tables.dtype == torch.int32 and token_seq.dtype == torch.int32
    assert positions.dtype == torch.int32 and keys.is_contiguous() and token_seq.shape[0] >= T and positions.shape[0] >= T
    out = torch.empty((T, S), dtype=torch.float32, device=q.device)
    rc = lib().xl_index_scores(_ptr(q), _ptr(w), _ptr(keys), _ptr(block_tables), _ptr(token_seq), _ptr(positions), _ptr(out),
                               c_int(T), c_int(S), c_int(block_tables.shape[0]), c_int(block_tables.shape[1]),
                               c_int(keys.shape[1]), c_long(keys.shape[0] * keys.shape[1]), c_int(NH), c_int(D), _stream())
    if rc == -3:
        return None
    _check(rc, "xl_index_scores")
    launch_count += 1
    return out


_ARANGE: Dict[Tuple[int, str], torch.Tensor] = {}


def mla_attention_sparse(q_lat_hm, q_pe_hm, cache, sel, sel_len, scale, kv_lora):
    """Head-major in and out.  Every query token is its own one-row sequence whose block table is its row of `sel`
    (blocks of one slot) and whose length is `sel_len[t]`: the paged MLA kernel then gathers exactly the kept rows."""
    global launch_count
    Hh, T, C = q_lat_hm.shape
    rope = q_pe_hm.shape[-1]
    if Hh % 16:
        raise RuntimeError(f"sparse MLA attention needs a multiple of 16 heads per rank (got {Hh})")
    key = (T + 1, str(q_lat_hm.device))
    q_cu = _ARANGE.get(key)
    if q_cu is None:
        q_cu = torch.arange(T + 1, dtype=torch.int32, device=q_lat_hm.device)
        if not torch.cuda.is_current_stream_capturing():      # a tensor made inside a capture lives in the graph's pool
            _ARANGE[key] = q_cu
    sel = sel.contiguous()
    sel_len = sel_len.contiguous()
    assert sel.dtype == torch.int32 and sel_len.dtype == torch.int32 and sel.shape[0] == T and sel_len.shape[0] == T
    out = torch.empty_like(q_lat_hm)
    rc = lib().xl_mla_attention(_ptr(q_lat_hm), _ptr(q_pe_hm), _ptr(cache), _ptr(out), _ptr(q_cu), _ptr(sel_len), _ptr(sel), c_int(0),
                                c_int(T), c_int(sel.shape[1]), c_int(1), c_long(cache.shape[0] * cache.shape[1]), c_int(Hh), c_int(T),
                                c_int(C), c_int(rope), c_float(scale), c_int(T * (Hh // 16)), _stream())
    _check(rc, "xl_mla_attention (sparse)")
    launch_count += 1
    return out


def mla_v_up(o_lat_hm, w_vc):
    """o_lat head-major [Hh, T, c] x W_vc [Hh, v, c] -> [T, Hh * v]."""
    from . import moe_cuda
    Hh, T, C = o_lat_hm.shape
    v = w_vc.shape[1]
    out = torch.empty((T, Hh * v), dtype=o_lat_hm.dtype, device=o_lat_hm.device)
    tiles = _HeadTiles.get(Hh, T, o_lat_hm.device)
    moe_cuda.grouped_gemm(o_lat_hm.view(Hh * T, C), w_vc, tiles, out=out, c_rows_per_expert=T, c_col_stride=v)
    return out


# ----------------------------------------------------------------------------- fp8 block-scaled
def quant_act_1x128(x: torch.Tensor, gated: bool = False, rows_dev: Optional[torch.Tensor] = None):
    """bf16 [T, K] -> (e4m3 [T, K], fp32 scales [T, K/128]).  gated: x is [T, 2K] = [gate | up], quantises silu(gate) * up."""
    global launch_count
    T = x.shape[0]
    K = x.shape[1] // (2 if gated else 1)
    if x.stride(-1) != 1:
        x = x.contiguous()
    q = torch.empty((T, K), dtype=torch.float8_e4m3fn, device=x.device)
    s = torch.empty((T, K // 128), dtype=torch.float32, device=x.device)
    _check(lib().xl_quant_act_1x128(_ptr(x), _ptr(q), _ptr(s), c_int(T), c_int(K), c_int(x.stride(0)), c_int(int(gated)),
                                    _ptr(rows_dev), _stream()), "xl_quant_act_1x128")
    launch_count += 1
    return q, s


def linear_fp8_block(x: torch.Tensor, wq: torch.Tensor, wscale: torch.Tensor, out_dtype=torch.bfloat16) -> torch.Tensor:
    global launch_count
    x2 = x.reshape(-1, x.shape[-1])
    M, K = x2.shape
    N = wq.shape[0]
    xq, xs = quant_act_1x128(x2)
    out = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
    _check(lib().xl_gemm_fp8_block(_ptr(xq), _ptr(wq), _ptr(out), _ptr(xs), _ptr(wscale), c_int(M), c_int(N), c_int(K),
                                   c_int(out.stride(0)), _stream()), "xl_gemm_fp8_block")
    launch_count += 1
    return out.reshape(x.shape[:-1] + (N,))


def moe_experts_fp8(x, w13, w13_scale, w2, w2_scale, weights, ids, expert_offset=0):
    """Routed experts with fp8 block-scaled weights: sort -> gather -> quant -> grouped fp8 GEMM -> SwiGLU+quant ->
    grouped fp8 GEMM -> combine."""
    global launch_count
    from . import moe_cuda
    T, H = x.shape
    k = ids.shape[1]
    E, I2, _ = w13.shape
    r = moe_cuda.moe_sort(ids, expert_offset, E)
    xs = moe_cuda.gather_rows(x, r, k)
    R = xs.shape[0]
    xq, xsc = quant_act_1x128(xs, rows_dev=r.total_rows)
    h = torch.empty((R, I2), dtype=torch.bfloat16, device=x.device)
    L = lib()
    _check(L.xl_grouped_gemm_fp8_block(_ptr(xq), _ptr(w13), _ptr(h), _ptr(xsc), _ptr(w13_scale), c_int(R), c_int(I2), c_int(H),
                                       c_int(h.stride(0)), c_int(E), _ptr(r.tile_expert), _ptr(r.tile_row0), _ptr(r.tile_row_end),
                                       _ptr(r.num_m_tiles), c_int(r.max_tiles), _stream()), "xl_grouped_gemm_fp8_block(w13)")
    hq, hsc = quant_act_1x128(h, gated=True, rows_dev=r.total_rows)
    y = torch.empty((R, H), dtype=torch.bfloat16, device=x.device)
    _check(L.xl_grouped_gemm_fp8_block(_ptr(hq), _ptr(w2), _ptr(y), _ptr(hsc), _ptr(w2_scale), c_int(R), c_int(H), c_int(I2 // 2),
                                       c_int(y.stride(0)), c_int(E), _ptr(r.tile_expert), _ptr(r.tile_row0), _ptr(r.tile_row_end),
                                       _ptr(r.num_m_tiles), c_int(r.max_tiles), _stream()), "xl_grouped_gemm_fp8_block(w2)")
    launch_count += 2
    return moe_cuda.combine(y, r, weights, T)


# ----------------------------------------------------------------------------- fp8 with per-row / per-channel scales
def _fp8_rows_out(T: int, H: int, device):
    return (torch.empty((T, H), dtype=torch.float8_e4m3fn, device=device), torch.empty((T,), dtype=torch.float32, device=device))


def quant_rows_fp8(x: torch.Tensor):
    """bf16 [T, H] -> (e4m3 [T, H], fp32 [T]): one dynamic scale per row (token)."""
    global launch_count
    if x.stride(-1) != 1:
        x = x.contiguous()
    T, H = x.shape
    q, s = _fp8_rows_out(T, H, x.device)
    _check(lib().xl_quant_rows_fp8(_ptr(x), _ptr(q), _ptr(s), c_int(T), c_int(H), c_int(x.stride(0)), _stream()), "xl_quant_rows_fp8")
    launch_count += 1
    return q, s


def rms_norm_quant_fp8(x: torch.Tensor, w: torch.Tensor, eps: float):
    global launch_count
    if x.stride(-1) != 1:
        x = x.contiguous()
    T, H = x.shape
    q, s = _fp8_rows_out(T, H, x.device)
    _check(lib().xl_rms_norm_quant_fp8(_ptr(x), _ptr(w), _ptr(q), _ptr(s), c_int(T), c_int(H), c_int(x.stride(0)), c_float(eps),
                                       _stream()), "xl_rms_norm_quant_fp8")
    launch_count += 1
    return q, s


def add_rms_norm_quant_fp8(x: torch.Tensor, residual: torch.Tensor, w: torch.Tensor, eps: float):
    """residual' = x + residual; returns (e4m3 RMSNorm(residual') * w, row scales, residual')."""
    global launch_count
    x, residual = x.contiguous(), residual.contiguous()
    T, H = x.shape
    q, s = _fp8_rows_out(T, H, x.device)
    res_out = torch.empty_like(residual)
    _check(lib().xl_add_rms_norm_quant_fp8(_ptr(x), _ptr(residual), _ptr(w), _ptr(q), _ptr(s), _ptr(res_out), c_int(T), c_int(H),
                                           c_float(eps), _stream()), "xl_add_rms_norm_quant_fp8")
    launch_count += 1
    return q, s, res_out


def linear_fp8_scaled(xq: torch.Tensor, xs: torch.Tensor, wq: torch.Tensor, col_scale: Optional[torch.Tensor] = None,
                      tensor_scale: float = 1.0, bias: Optional[torch.Tensor] = None, swiglu: bool = False) -> torch.Tensor:
    """bf16 [M, N] = (xq wq^T) * xs[m] * tensor_scale * col_scale[n] (+ bias); `swiglu`: wq holds interleaved gate / up rows
    (as `interleave_gate_up` lays them out, `col_scale` in the same order) and the result is silu(gate) * up [M, N / 2]."""
    global launch_count
    M, K = xq.shape
    N = wq.shape[0]
    assert xq.dtype == torch.float8_e4m3fn and wq.dtype == torch.float8_e4m3fn and wq.shape[1] == K and xq.stride(-1) == 1
    out = torch.empty((M, N // 2 if swiglu else N), dtype=torch.bfloat16, device=xq.device)
    if M > 0:
        epi = 2 if swiglu else (1 if bias is not None else 0)
        assert not (swiglu and bias is not None)
        _check(lib().xl_gemm_fp8_scaled(c_int(epi), _ptr(xq), _ptr(wq), _ptr(out), _ptr(bias), _ptr(xs), _ptr(col_scale),
                                        c_float(tensor_scale), c_int(M), c_int(N), c_int(K), c_int(xq.stride(0)), c_int(wq.stride(0)),
                                        c_int(out.stride(0)), _stream()), "xl_gemm_fp8_scaled")
        launch_count += 1
    return out
