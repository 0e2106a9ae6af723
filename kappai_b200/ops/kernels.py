"""Python faces of the CUDA kernels.

Each function checks its tensors (device, dtype, layout), launches on the
current CUDA stream and raises on any error.  There is no CPU path: a tensor
that is not on a CUDA device is refused.
"""
from __future__ import annotations

import ctypes
from typing import Optional, Tuple

import torch

from .build import is_loaded, load_library

F32, BF16 = 0, 1
EPI_STORE, EPI_STORE_F32, EPI_ACCUM_F32 = 0, 1, 2


MAX_STEP_ROWS = 65535     # rows of one step: the row-wise kernels put rows on a grid axis that ends there

LAUNCHES = [0]      # kernel launchers called so far (a launcher may launch more than one kernel)
LAUNCHES_BY = {}    # the same by launcher name


class KernelError(RuntimeError):
    pass


def dtype_code(dt: torch.dtype) -> int:
    if dt == torch.float32:
        return F32
    if dt == torch.bfloat16:
        return BF16
    raise KernelError(f"kernels take float32 or bfloat16 tensors, got {dt}")


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)
_raw_device = getattr(torch._C, "_cuda_getDevice", None)


def _stream() -> ctypes.c_void_p:
    """The current CUDA stream of the current device (asked of torch's C layer directly where it offers that:
    this runs once per kernel launch)."""
    if _raw_stream is not None and _raw_device is not None:
        return ctypes.c_void_p(_raw_stream(_raw_device()))
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


def _ptr(t: Optional[torch.Tensor]) -> ctypes.c_void_p:
    return ctypes.c_void_p(0 if t is None else t.data_ptr())


def _need(t: torch.Tensor, name: str, dtype=None, contiguous: bool = True) -> None:
    if not isinstance(t, torch.Tensor) or not t.is_cuda:
        raise KernelError(f"{name}: expected a CUDA tensor (kappai_b200 has no CPU path)")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{name}: expected {dtype}, got {t.dtype}")
    if contiguous and not t.is_contiguous():
        raise KernelError(f"{name}: expected a contiguous tensor")


class _Stream:
    """Stands for "the current stream" among a launcher's arguments."""


STREAM = _Stream()


class KernelTimer:
    """Device time by kernel class: while one is installed (``TIMER[0]``), every launcher call is put between
    two CUDA events on its stream; ``report`` adds them up by class.  The reference keeps per-stage counters of
    the same kind (src/profile.h:9-47,77-88) and prints them with ``--time`` (src/profile.c:65-110).  A class is
    the launcher's name, for matrix products with the weight's shape.  Only launches made one by one are seen:
    the engine runs its steps eagerly (no captured graphs) while it is timed, so the times of small kernels
    include the gap the host leaves before them."""

    FOLD_AT = 8192

    def __init__(self):
        self._open = []                    # (class, event before, event after, flops, bytes)
        self.totals = {}                   # class -> [calls, ms, flops, bytes]

    def add(self, key, e0, e1, work) -> None:
        self._open.append((key, e0, e1, work))
        if len(self._open) >= self.FOLD_AT:
            self.fold()

    def fold(self) -> None:
        if not self._open:
            return
        self._open[-1][2].synchronize()
        for key, e0, e1, work in self._open:
            t = self.totals.setdefault(key, [0, 0.0, 0, 0])
            t[0] += 1
            t[1] += e0.elapsed_time(e1)
            if work:
                t[2] += work[0]
                t[3] += work[1]
        self._open = []

    def report(self):
        """Rows (class, calls, ms, microseconds a call, share in per cent, TFLOP/s or None, GB/s or None),
        the class that took longest first."""
        self.fold()
        total = sum(t[1] for t in self.totals.values()) or 1.0
        rows = []
        for key, (calls, ms, flops, nbytes) in sorted(self.totals.items(), key=lambda kv: -kv[1][1]):
            rows.append((key, calls, ms, ms * 1e3 / calls, 100.0 * ms / total,
                         flops / (ms * 1e-3) / 1e12 if flops and ms > 0 else None,
                         nbytes / (ms * 1e-3) / 1e9 if nbytes and ms > 0 else None))
        return rows

    def format(self, label: str = "kernels") -> str:
        rows = self.report()
        total = sum(r[2] for r in rows)
        out = [f"[profile] {label}  accounted={total * 1e3:.0f} us",
               f"  {'class':<34} {'ms':>10} {'calls':>8} {'us/call':>9} {'share':>7} {'TFLOP/s':>8} {'GB/s':>8}"]
        for key, calls, ms, per, share, tf, gb in rows:
            out.append(f"  {key:<34} {ms:>10.3f} {calls:>8d} {per:>9.2f} {share:>6.2f}% "
                       f"{'' if tf is None else format(tf, '8.1f'):>8} {'' if gb is None else format(gb, '8.1f'):>8}")
        return "\n".join(out)


TIMER = [None]         # the KernelTimer that watches the launches, if any


def _run(what: str, fn, *args, tag: str = "", work=None) -> None:
    """The one door to the kernel libraries: call the launcher ``fn`` on the current stream and check its
    answer.  ``tag`` and ``work`` = (flops, bytes) describe the call to a :class:`KernelTimer`."""
    timer = TIMER[0]
    if timer is None:
        _check(fn(*[_stream() if a is STREAM else a for a in args]), what)
        if LAUNCH_LOG[0] is not None and tag:
            LAUNCH_LOG[0][-1] += tag
        return
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    _check(fn(*[_stream() if a is STREAM else a for a in args]), what)
    e1.record()
    timer.add(what + tag, e0, e1, work)


def _gemm_work(M: int, N: int, K: int, a: torch.Tensor, w: torch.Tensor, out: torch.Tensor):
    return (2 * M * N * K, M * K * a.element_size() + N * K * w.element_size() + out.numel() * out.element_size())


LAUNCH_LOG = [None]        # a list: every launch appends its name (bench.py --probe timeline names a step's kernels by it)


def _check(status: int, what: str) -> None:
    LAUNCHES[0] += 1
    LAUNCHES_BY[what] = LAUNCHES_BY.get(what, 0) + 1
    if LAUNCH_LOG[0] is not None:
        LAUNCH_LOG[0].append(what)
    if status != 0:
        if status == -95:
            raise KernelError(f"{what}: size not supported by this kernel")
        if status == -22:
            raise KernelError(f"{what}: bad argument")
        raise KernelError(f"{what}: CUDA error {status}")


def _rows_2d(t: torch.Tensor, name: str) -> int:
    """Leading dimension (in elements) of a 2-D tensor whose rows are contiguous."""
    if t.dim() != 2 or t.stride(1) != 1:
        raise KernelError(f"{name}: expected a 2-D tensor with contiguous rows")
    return t.stride(0)


# --------------------------------------------------------------- status words
# Kernels that wait on a barrier wait with a limit; one that gives up sets its library's status word, stops
# issuing work and returns.  The engine reads the words of a step with the step's own device-to-host copy.

_STATUS_LIBS = (("gemm_tc", "tc"), ("gemm_stream", "stream"), ("attention_mma", "attention_mma"),
                ("attention_tc", "attention_tc"), ("moe", "moe_tc"), ("latent", "latent"))


def read_status() -> dict:
    """Library -> status word (0, or 1 if a bounded wait gave up since the last call) of every kernel library
    that is loaded and has one; the words are cleared.  Synchronises the device."""
    return {lib: _read_one(lib, name) for lib, name in _STATUS_LIBS if is_loaded(lib)}


def _read_one(lib: str, name: str) -> int:
    return int(getattr(load_library(lib), f"kp_{name}_status")()) if is_loaded(lib) else 0


def tc_status() -> int:
    """0, or 1 if a bounded wait of the tcgen05 product kernel gave up since the last call (synchronises)."""
    return _read_one("gemm_tc", "tc")


def stream_status() -> int:
    return _read_one("gemm_stream", "stream")


def attention_tc_status() -> int:
    return _read_one("attention_tc", "attention_tc")


def attention_mma_status() -> int:
    return _read_one("attention_mma", "attention_mma")


class StatusGather:
    """Collects the status words of the loaded kernel libraries (and one word of its own, ``injected``, that
    the host may set: a stand-in for a kernel failure where the real one cannot be made) into one device
    word, with one small kernel behind a step."""

    def __init__(self, device: torch.device):
        self.device = device
        self.injected = torch.zeros(1, dtype=torch.int32, device=device)
        self._libs = None
        self._addrs: Optional[torch.Tensor] = None

    def _refresh(self) -> None:
        libs = tuple(lib for lib, _ in _STATUS_LIBS if is_loaded(lib))
        if libs == self._libs:
            return
        addrs = [self.injected.data_ptr()]
        for lib, name in _STATUS_LIBS:
            if lib in libs:
                fn = getattr(load_library(lib), f"kp_{name}_status_address")
                fn.restype = ctypes.c_void_p
                a = fn()
                if not a:
                    raise KernelError(f"{lib}: no address for its status word")
                addrs.append(int(a))
        self._addrs = torch.tensor(addrs, dtype=torch.int64).to(self.device)
        self._libs = libs

    def gather(self, out: torch.Tensor) -> None:
        """out[0] (int32, on the device) = OR of the status words, in stream order."""
        _need(out, "out", torch.int32)
        self._refresh()
        _run("gather_status", load_library("rowwise").kp_gather_status, _ptr(self._addrs), self._addrs.numel(), _ptr(out), STREAM)

    def clear(self) -> dict:
        """Read and clear every word (synchronises); returns what was set."""
        st = read_status()
        if int(self.injected.item()):
            st["injected"] = 1
            self.injected.zero_()
        return {k: v for k, v in st.items() if v}


# -------------------------------------------------------------------- rowwise

def step_tables(src_pinned: torch.Tensor, dst: torch.Tensor, tokens: Optional[torch.Tensor] = None, tok_off: int = 0) -> None:
    """The int32 tables of a captured step from their staging buffer in pinned host memory to the device buffer
    ``dst`` by a kernel (the device reads the host buffer itself), and with them ``tokens`` (int32, on the device)
    to words ``tok_off`` ... of ``dst``."""
    if src_pinned.dtype != torch.int32 or not src_pinned.is_pinned() or src_pinned.numel() != dst.numel():
        raise KernelError("step_tables: the source is an int32 tensor in pinned memory, as long as the destination")
    _need(dst, "dst", torch.int32)
    n_tok = 0
    if tokens is not None:
        _need(tokens, "tokens", torch.int32)
        n_tok = tokens.numel()
    _run("step_tables", load_library("rowwise").kp_step_tables, ctypes.c_void_p(src_pinned.data_ptr()), _ptr(dst), dst.numel(),
         _ptr(tokens), tok_off, n_tok, STREAM)


def embed_rows(table: torch.Tensor, ids: torch.Tensor, out: torch.Tensor, scale: float = 1.0,
               pos_table: Optional[torch.Tensor] = None, positions: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[r] = table[ids[r]] * scale (+ pos_table[positions[r]], a table of learned position vectors)."""
    _need(table, "table"); _need(ids, "ids", torch.int32); _need(out, "out", torch.float32)
    n, d = out.shape
    if table.shape[1] != d or ids.numel() != n:
        raise KernelError("embed_rows: shape mismatch")
    if pos_table is not None:
        _need(pos_table, "pos_table", table.dtype); _need(positions, "positions", torch.int32)
        if pos_table.shape[1] != d or positions.numel() != n:
            raise KernelError("embed_rows: position table shape mismatch")
    lib = load_library("rowwise")
    _run("embed_rows", lib.kp_embed_rows, _ptr(table), _ptr(ids), _ptr(out), n, d, ctypes.c_float(scale),
         _ptr(pos_table), _ptr(positions if pos_table is not None else None), dtype_code(table.dtype), STREAM)
    return out


def rmsnorm_rows(x: torch.Tensor, w: torch.Tensor, eps: float, out: torch.Tensor,
                 rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[r] = rmsnorm(x[rows[r]] if rows is given else x[r])."""
    _need(x, "x", torch.float32); _need(w, "w", torch.float32); _need(out, "out")
    n, d = out.shape
    if x.shape[1] != d or w.numel() != d:
        raise KernelError("rmsnorm_rows: shape mismatch")
    if rows is not None:
        _need(rows, "rows", torch.int32)
        if rows.numel() != n:
            raise KernelError("rmsnorm_rows: rows/out mismatch")
    elif x.shape[0] != n:
        raise KernelError("rmsnorm_rows: x/out mismatch")
    lib = load_library("rowwise")
    _run("rmsnorm_rows", lib.kp_rmsnorm_rows, _ptr(x), _ptr(w), _ptr(out), _ptr(rows), n, d, ctypes.c_float(eps),
                               dtype_code(out.dtype), STREAM)
    return out


def layernorm_rows(x: torch.Tensor, w: torch.Tensor, eps: float, out: torch.Tensor,
                   rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[r] = (x - mean) / sqrt(var + eps) * w of the float32 row x[rows[r]] (x[r] without ``rows``): a weighted layer
    norm without a shift, the variance taken about the mean."""
    _need(x, "x", torch.float32); _need(w, "w", torch.float32); _need(out, "out")
    n, d = out.shape
    if x.shape[1] != d or w.numel() != d:
        raise KernelError("layernorm_rows: shape mismatch")
    if rows is not None:
        _need(rows, "rows", torch.int32)
        if rows.numel() != n:
            raise KernelError("layernorm_rows: rows/out mismatch")
    elif x.shape[0] != n:
        raise KernelError("layernorm_rows: x/out mismatch")
    if n > MAX_STEP_ROWS:
        raise KernelError("layernorm_rows: too many rows")
    _run("layernorm_rows", load_library("rowwise").kp_layernorm_rows, _ptr(x), _ptr(w), _ptr(out), _ptr(rows), n, d,
         ctypes.c_float(eps), dtype_code(out.dtype), STREAM)
    return out


GATE_ACTS = {"silu": 0, "sigmoid": 1}


def group_norm_gate_rows(o: torch.Tensor, w: Optional[torch.Tensor], g: torch.Tensor, eps: float, out: torch.Tensor,
                         groups: int, gate_first: bool, gate_act: str = "silu") -> torch.Tensor:
    """The float32 rows ``o`` [n, c] RMS-normed in ``groups`` stretches of equal width (a mean square a stretch), with a
    gate ``act(g)`` (silu or sigmoid; ``g`` [n, c] in the storage type, rows may be strided) and an optional weight
    ``w`` [c]: ``gate_first`` -> ``norm(o * act(g)) * w``, else ``norm(o) * w * act(g)``."""
    _need(o, "o", torch.float32); _need(out, "out"); _need(g, "g", out.dtype, contiguous=False)
    n, c = o.shape
    if tuple(out.shape) != (n, c) or tuple(g.shape) != (n, c) or groups < 1 or c % groups:
        raise KernelError("group_norm_gate_rows: shape mismatch")
    if w is not None:
        _need(w, "w", torch.float32)
        if w.numel() != c:
            raise KernelError("group_norm_gate_rows: weight size")
    if gate_act not in GATE_ACTS:
        raise KernelError(f"group_norm_gate_rows: gate '{gate_act}' (silu or sigmoid)")
    if n > MAX_STEP_ROWS:
        raise KernelError("group_norm_gate_rows: too many rows")
    _run("group_norm_gate_rows", load_library("rowwise").kp_group_norm_gate_rows, _ptr(o), c, _ptr(w), _ptr(g), _rows_2d(g, "g"),
         _ptr(out), c, n, int(groups), c // int(groups), ctypes.c_float(eps), int(bool(gate_first)), GATE_ACTS[gate_act],
         dtype_code(out.dtype), STREAM)
    return out


def head_gate(o: torch.Tensor, g: torch.Tensor, H: int, hd: int) -> torch.Tensor:
    """o[r, h hd + i] *= sigmoid(g[r, h]) in place: one gate a head (``g`` [n, H], rows may be strided)."""
    _need(o, "o"); _need(g, "g", o.dtype, contiguous=False)
    n = o.shape[0]
    if tuple(o.shape) != (n, H * hd) or tuple(g.shape) != (n, H):
        raise KernelError("head_gate: shape mismatch")
    _run("head_gate", load_library("rowwise").kp_head_gate, _ptr(o), H * hd, _ptr(g), _rows_2d(g, "g"), n, H, hd,
         dtype_code(o.dtype), STREAM)
    return o


def softcap(x: torch.Tensor, cap: float) -> torch.Tensor:
    """x <- cap * tanh(x / cap) in place (float32)."""
    _need(x, "x", torch.float32)
    if not cap > 0:
        raise KernelError("softcap: the cap must be positive")
    _run("softcap", load_library("rowwise").kp_softcap, _ptr(x), ctypes.c_longlong(x.numel()), ctypes.c_float(cap), STREAM)
    return x


def glu_clamped(gate_up: torch.Tensor, out: torch.Tensor, limit: float, alpha: float, shift: float) -> torch.Tensor:
    """out = g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit), rows [gate | up]."""
    _need(gate_up, "gate_up"); _need(out, "out", gate_up.dtype)
    n, ff = out.shape
    if gate_up.shape != (n, 2 * ff):
        raise KernelError("glu_clamped: shape mismatch")
    _run("glu_clamped", load_library("rowwise").kp_glu_clamped, _ptr(gate_up), _ptr(out), n, ff, ctypes.c_float(limit),
         ctypes.c_float(alpha), ctypes.c_float(shift), dtype_code(out.dtype), STREAM)
    return out


ACTIVATIONS = {"silu": 0, "relu": 1, "gelu_tanh": 2}     # codes of the gated units' activations (csrc/common.cuh)


PLAIN_ACTIVATIONS = dict(ACTIVATIONS, relu_squared=4)    # the ungated units have one more


def plain_activation_code(name: str) -> int:
    if name not in PLAIN_ACTIVATIONS:
        raise KernelError(f"activation '{name}' (expected one of {', '.join(PLAIN_ACTIVATIONS)})")
    return PLAIN_ACTIVATIONS[name]


def activation_code(name: str) -> int:
    try:
        return ACTIVATIONS[name]
    except KeyError:
        raise KernelError(f"activation '{name}': expected one of {', '.join(ACTIVATIONS)}") from None


def swiglu(gate_up: torch.Tensor, out: torch.Tensor, activation: str = "silu") -> torch.Tensor:
    """out = act(gate) * up for rows [gate | up]."""
    _need(gate_up, "gate_up"); _need(out, "out", gate_up.dtype)
    n, ff = out.shape
    if gate_up.shape != (n, 2 * ff):
        raise KernelError("swiglu: shape mismatch")
    lib = load_library("rowwise")
    _run("swiglu", lib.kp_swiglu, _ptr(gate_up), _ptr(out), n, ff, activation_code(activation), dtype_code(out.dtype), STREAM)
    return out


def postnorm_rows(acc: torch.Tensor, w: torch.Tensor, eps: float, x_out: Optional[torch.Tensor] = None,
                  h_out: Optional[torch.Tensor] = None, scaled_out: Optional[torch.Tensor] = None,
                  alpha: float = 1.0) -> None:
    """y = rmsnorm(acc) * w for the float32 rows of ``acc``; y goes to ``x_out`` (float32), ``h_out`` (any
    storage type) and, times ``alpha``, to ``scaled_out`` (float32), whichever are given (each may be ``acc``)."""
    _need(acc, "acc", torch.float32); _need(w, "w", torch.float32)
    n, d = acc.shape
    if w.numel() != d:
        raise KernelError("postnorm_rows: weight size")
    for t, nm, dt in ((x_out, "x_out", torch.float32), (h_out, "h_out", None), (scaled_out, "scaled_out", torch.float32)):
        if t is not None:
            _need(t, nm, dt)
            if tuple(t.shape) != (n, d):
                raise KernelError(f"postnorm_rows: {nm} shape")
    if n > MAX_STEP_ROWS:
        raise KernelError("postnorm_rows: too many rows")
    code = dtype_code(h_out.dtype) if h_out is not None else F32
    _run("postnorm_rows", load_library("rowwise").kp_postnorm_rows, _ptr(acc), _ptr(w), _ptr(x_out), _ptr(h_out),
         _ptr(scaled_out), n, d, ctypes.c_float(eps), ctypes.c_float(alpha), code, STREAM)


def scale_cast(x: torch.Tensor, h_out: Optional[torch.Tensor], scaled_out: torch.Tensor, alpha: float) -> None:
    """h_out = x in h_out's type (if given), scaled_out = alpha * x (float32)."""
    _need(x, "x", torch.float32); _need(scaled_out, "scaled_out", torch.float32)
    if h_out is not None:
        _need(h_out, "h_out")
        if h_out.numel() != x.numel():
            raise KernelError("scale_cast: size mismatch")
    if scaled_out.numel() != x.numel():
        raise KernelError("scale_cast: size mismatch")
    code = dtype_code(h_out.dtype) if h_out is not None else F32
    _run("scale_cast", load_library("rowwise").kp_scale_cast, _ptr(x), _ptr(h_out), _ptr(scaled_out),
         ctypes.c_longlong(x.numel()), ctypes.c_float(alpha), code, STREAM)


def sigmoid_gate(o: torch.Tensor, g: torch.Tensor) -> torch.Tensor:
    """o *= sigmoid(g), element by element; both 2-D with contiguous rows (``g`` may be columns of a wider tensor)."""
    _need(o, "o", contiguous=False); _need(g, "g", o.dtype, contiguous=False)
    if o.shape != g.shape:
        raise KernelError("sigmoid_gate: shape mismatch")
    _run("sigmoid_gate", load_library("rowwise").kp_sigmoid_gate, _ptr(o), _rows_2d(o, "o"), _ptr(g), _rows_2d(g, "g"),
         o.shape[0], o.shape[1], dtype_code(o.dtype), STREAM)
    return o


def rmsnorm_cols(x: torch.Tensor, stretches, eps: float) -> None:
    """RMS norm of one or two column stretches of the rows of ``x`` (storage type), each on its own:
    ``stretches`` = [(first column, weight float32 [width], out [n, width] in x's type), ...]."""
    _need(x, "x", contiguous=False)
    if not 1 <= len(stretches) <= 2:
        raise KernelError("rmsnorm_cols: one or two stretches")
    n = x.shape[0]
    args = []
    for col, w, out in stretches:
        _need(w, "weight", torch.float32); _need(out, "out", x.dtype, contiguous=False)
        width = w.numel()
        if col < 0 or col + width > x.shape[1] or tuple(out.shape) != (n, width):
            raise KernelError("rmsnorm_cols: shape mismatch")
        args += [int(col), width, _ptr(w), _ptr(out), _rows_2d(out, "out")]
    if len(stretches) == 1:
        args += [0, 0, _ptr(None), _ptr(None), 0]
    _run("rmsnorm_cols", load_library("rowwise").kp_rmsnorm_cols, _ptr(x), _rows_2d(x, "x"), n, ctypes.c_float(eps), *args,
         dtype_code(x.dtype), STREAM)


def norm_gate_rows(o: torch.Tensor, w: torch.Tensor, g: torch.Tensor, eps: float, out: torch.Tensor) -> torch.Tensor:
    """out = rmsnorm(o) * w * sigmoid(g): float32 rows ``o`` normed whole, gated by columns ``g`` of a wider row."""
    _need(o, "o", torch.float32); _need(w, "w", torch.float32); _need(g, "g", contiguous=False)
    _need(out, "out", g.dtype, contiguous=False)
    n, d = o.shape
    if w.numel() != d or tuple(g.shape) != (n, d) or tuple(out.shape) != (n, d):
        raise KernelError("norm_gate_rows: shape mismatch")
    _run("norm_gate_rows", load_library("rowwise").kp_norm_gate_rows, _ptr(o), _ptr(w), _ptr(g), _rows_2d(g, "g"), _ptr(out),
         _rows_2d(out, "out"), n, d, ctypes.c_float(eps), dtype_code(g.dtype), STREAM)
    return out


def token_gate(gate: torch.Tensor, table: torch.Tensor, col0: int, ids: torch.Tensor, out: torch.Tensor,
               activation: str = "gelu_tanh") -> torch.Tensor:
    """out[r, c] = act(gate[r, c]) * table[ids[r], col0 + c]."""
    _need(gate, "gate", contiguous=False); _need(table, "table", gate.dtype, contiguous=False)
    _need(ids, "ids", torch.int32); _need(out, "out", gate.dtype)
    n, dim = gate.shape
    if tuple(out.shape) != (n, dim) or ids.numel() != n or col0 < 0 or col0 + dim > table.shape[1]:
        raise KernelError("token_gate: shape mismatch")
    _run("token_gate", load_library("rowwise").kp_token_gate, _ptr(gate), _rows_2d(gate, "gate"), _ptr(table),
         _rows_2d(table, "table"), int(col0), _ptr(ids), _ptr(out), n, dim, activation_code(activation),
         dtype_code(gate.dtype), STREAM)
    return out


def rmsnorm_add_rows(y: torch.Tensor, w: torch.Tensor, eps: float, x: torch.Tensor) -> torch.Tensor:
    """x += rmsnorm(y) * w (all float32)."""
    _need(y, "y", torch.float32); _need(w, "w", torch.float32); _need(x, "x", torch.float32)
    n, d = x.shape
    if tuple(y.shape) != (n, d) or w.numel() != d:
        raise KernelError("rmsnorm_add_rows: shape mismatch")
    _run("rmsnorm_add_rows", load_library("rowwise").kp_rmsnorm_add_rows, _ptr(y), _ptr(w), _ptr(x), n, d, ctypes.c_float(eps), STREAM)
    return x


def rmsnorm_add_norm_rows(y: torch.Tensor, w_branch: torch.Tensor, eps_branch: float, x: torch.Tensor,
                          w_next: Optional[torch.Tensor] = None, eps_next: float = 0.0,
                          h_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x += rmsnorm(y) * w_branch (float32), y cleared; with ``w_next`` and ``h_out`` also
    ``h_out = rmsnorm(x) * w_next`` of the new x, in ``h_out``'s type: the norms behind one sublayer and in front
    of the next in one launch."""
    _need(y, "y", torch.float32); _need(w_branch, "w_branch", torch.float32); _need(x, "x", torch.float32)
    n, d = x.shape
    if tuple(y.shape) != (n, d) or w_branch.numel() != d or (w_next is None) != (h_out is None):
        raise KernelError("rmsnorm_add_norm_rows: shape mismatch")
    if n > MAX_STEP_ROWS:
        raise KernelError("rmsnorm_add_norm_rows: too many rows")
    if h_out is not None:
        _need(w_next, "w_next", torch.float32); _need(h_out, "h_out")
        if tuple(h_out.shape) != (n, d) or w_next.numel() != d:
            raise KernelError("rmsnorm_add_norm_rows: shape mismatch")
    _run("rmsnorm_add_norm_rows", load_library("rowwise").kp_rmsnorm_add_norm_rows, _ptr(y), _ptr(w_branch),
         ctypes.c_float(eps_branch), _ptr(x), _ptr(w_next), ctypes.c_float(eps_next), _ptr(h_out), n, d,
         dtype_code(h_out.dtype if h_out is not None else torch.float32), STREAM)
    return x


def gated_add_norm_rows(y: torch.Tensor, gate: Optional[torch.Tensor], scale: Optional[torch.Tensor], x: torch.Tensor,
                        w_next: Optional[torch.Tensor] = None, eps_next: float = 0.0,
                        h_out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x += scale * sigmoid(gate) * y (float32; ``scale`` [d] or None: 1, ``gate`` [n, d] in the compute type, its rows may be
    strided, or None: 1), y cleared; with ``w_next`` and ``h_out`` also ``h_out = rmsnorm(x) * w_next`` of the new x."""
    _need(y, "y", torch.float32); _need(x, "x", torch.float32)
    n, d = x.shape
    if tuple(y.shape) != (n, d) or (w_next is None) != (h_out is None):
        raise KernelError("gated_add_norm_rows: shape mismatch")
    dt = gate.dtype if gate is not None else (h_out.dtype if h_out is not None else torch.float32)
    if gate is not None:
        _need(gate, "gate", contiguous=False)
        if tuple(gate.shape) != (n, d):
            raise KernelError("gated_add_norm_rows: gate shape")
    if scale is not None:
        _need(scale, "scale", torch.float32)
        if scale.numel() != d:
            raise KernelError("gated_add_norm_rows: scale size")
    if h_out is not None:
        _need(w_next, "w_next", torch.float32); _need(h_out, "h_out", dt)
        if tuple(h_out.shape) != (n, d) or w_next.numel() != d:
            raise KernelError("gated_add_norm_rows: shape mismatch")
    if n > MAX_STEP_ROWS:
        raise KernelError("gated_add_norm_rows: too many rows")
    _run("gated_add_norm_rows", load_library("rowwise").kp_gated_add_norm_rows, _ptr(y), _ptr(gate),
         _rows_2d(gate, "gate") if gate is not None else 0, _ptr(scale), _ptr(x), _ptr(w_next), ctypes.c_float(eps_next), _ptr(h_out),
         n, d, dtype_code(dt), STREAM,
         work=(0, n * d * (16 + (gate.element_size() if gate is not None else 0) + (h_out.element_size() if h_out is not None else 0))))
    return x


def activate(x: torch.Tensor, out: torch.Tensor, activation: str) -> torch.Tensor:
    """out = act(x), element by element (float32 in, ``out`` in the compute type)."""
    _need(x, "x", torch.float32); _need(out, "out")
    if x.shape != out.shape:
        raise KernelError("activate: shape mismatch")
    _run("activate", load_library("rowwise").kp_activate, _ptr(x), _ptr(out), ctypes.c_longlong(x.numel()), plain_activation_code(activation),
         dtype_code(out.dtype), STREAM)
    return out


def row_gate_add(h: torch.Tensor, w_gate: torch.Tensor, y: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """out[r] += sigmoid(h[r] . w_gate) * y[r]: ``w_gate`` float32 [d], ``y`` and ``out`` float32 [n, d]."""
    _need(h, "h", contiguous=False); _need(w_gate, "w_gate", torch.float32); _need(y, "y", torch.float32)
    _need(out, "out", torch.float32)
    n, d = h.shape
    if w_gate.numel() != d or tuple(y.shape) != (n, d) or tuple(out.shape) != (n, d):
        raise KernelError("row_gate_add: shape mismatch")
    _run("row_gate_add", load_library("rowwise").kp_row_gate_add, _ptr(h), _rows_2d(h, "h"), _ptr(w_gate), _ptr(y), _ptr(out),
         n, d, dtype_code(h.dtype), STREAM)
    return out


def cast(src: torch.Tensor, dst: torch.Tensor) -> torch.Tensor:
    _need(src, "src"); _need(dst, "dst")
    if src.numel() != dst.numel():
        raise KernelError("cast: size mismatch")
    lib = load_library("rowwise")
    _run("cast", lib.kp_cast, _ptr(src), _ptr(dst), ctypes.c_longlong(src.numel()), dtype_code(src.dtype),
                       dtype_code(dst.dtype), STREAM)
    return dst


# ----------------------------------------------------------------------- gemm

def gemm_nt_simt(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: Optional[torch.Tensor] = None,
                 accumulate: bool = False) -> torch.Tensor:
    """out = a @ w.T (+ bias); with ``accumulate`` out (float32) += that."""
    _need(a, "a", contiguous=False); _need(w, "w", a.dtype, contiguous=False); _need(out, "out", contiguous=False)
    lda, ldw, ldc = _rows_2d(a, "a"), _rows_2d(w, "w"), _rows_2d(out, "out")
    M, K = a.shape
    N = w.shape[0]
    if w.shape[1] != K or out.shape != (M, N):
        raise KernelError(f"gemm: shapes a{tuple(a.shape)} w{tuple(w.shape)} out{tuple(out.shape)} do not agree")
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() != N:
            raise KernelError("gemm: bias size")
    if accumulate:
        if out.dtype != torch.float32:
            raise KernelError("gemm: accumulation needs a float32 output")
        epi = EPI_ACCUM_F32
    elif out.dtype == a.dtype:
        epi = EPI_STORE
    elif out.dtype == torch.float32:
        epi = EPI_STORE_F32
    else:
        raise KernelError("gemm: output dtype must be the operand dtype or float32")
    lib = load_library("gemm_simt")
    _run("gemm_nt_simt", lib.kp_gemm_nt_simt, _ptr(a), _ptr(w), _ptr(bias), _ptr(out), M, N, K, lda, ldw, ldc, epi,
         dtype_code(a.dtype), STREAM, tag=f" {N}x{K}", work=_gemm_work(M, N, K, a, w, out))
    return out


# ------------------------------------------------------------------ shortconv

def shortconv_forward(p: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor,
                      row_seg: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor,
                      seg_slot: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    _need(p, "p", contiguous=False); _need(w, "w", torch.float32); _need(state, "state", torch.float32)
    _need(out, "out", p.dtype, contiguous=False)
    for t, nm in ((row_seg, "row_seg"), (cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    n, d = out.shape
    K = w.shape[1]
    if p.shape != (n, 3 * d) or w.shape[0] != d or state.shape[1:] != (K - 1, d):
        raise KernelError("shortconv_forward: shape mismatch")
    if bias is not None:
        _need(bias, "bias", torch.float32)
    lib = load_library("shortconv")
    _run("shortconv_forward", lib.kp_shortconv_forward, _ptr(p), _rows_2d(p, "p"), _ptr(w), _ptr(bias), _ptr(state), _ptr(row_seg),
                                    _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(out), _rows_2d(out, "out"),
                                    n, d, K, dtype_code(p.dtype), STREAM)
    return out


def shortconv_decode(p: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor,
                     seg_pos: torch.Tensor, seg_slot: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """Output and state update in one launch, for steps in which every segment is one row."""
    _need(p, "p", contiguous=False); _need(w, "w", torch.float32); _need(state, "state", torch.float32)
    _need(out, "out", p.dtype, contiguous=False)
    _need(seg_pos, "seg_pos", torch.int32); _need(seg_slot, "seg_slot", torch.int32)
    n, d = out.shape
    K = w.shape[1]
    if p.shape != (n, 3 * d) or w.shape[0] != d or state.shape[1:] != (K - 1, d) or seg_pos.numel() != n:
        raise KernelError("shortconv_decode: shape mismatch")
    if bias is not None:
        _need(bias, "bias", torch.float32)
    lib = load_library("shortconv")
    _run("shortconv_decode", lib.kp_shortconv_decode, _ptr(p), _rows_2d(p, "p"), _ptr(w), _ptr(bias), _ptr(state), _ptr(seg_pos),
                                   _ptr(seg_slot), _ptr(out), _rows_2d(out, "out"), n, d, K, dtype_code(p.dtype),
                                   STREAM)
    return out


def shortconv_update_state(p: torch.Tensor, state: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor,
                           seg_slot: torch.Tensor, n_seg: int) -> None:
    _need(p, "p", contiguous=False); _need(state, "state", torch.float32)
    d = p.shape[1] // 3
    K = state.shape[1] + 1
    if state.shape[2] != d:
        raise KernelError("shortconv_update_state: shape mismatch")
    lib = load_library("shortconv")
    _run("shortconv_update_state", lib.kp_shortconv_update_state, _ptr(p), _rows_2d(p, "p"), _ptr(state), _ptr(cu_rows), _ptr(seg_pos),
                                         _ptr(seg_slot), n_seg, d, K, dtype_code(p.dtype), STREAM)


# ------------------------------------------------------------------ linear attention with decay

LIGHTNING_MAX_DIM = 256    # key rows of a head's state that the scan keeps in registers


def lightning_scan(qkv: torch.Tensor, q_col: int, k_col: int, v_col: int, decay_hi: torch.Tensor, decay_lo: torch.Tensor,
                   state: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor, seg_slot: torch.Tensor,
                   out: torch.Tensor, n_seg: int, H: int, dim: int, vdim: int, activation: Optional[str] = "silu",
                   write_state: bool = True, rotary=None, k_scale: float = 1.0) -> torch.Tensor:
    """``S <- a_h S + k v^T; o = S^T q`` row after row of every segment, from the state in the segment's slot (zero at
    position 0) and back into it.  q, k (H heads of ``dim``) and v (H heads of ``vdim``) are columns of ``qkv`` in
    the storage type with ``activation`` (silu or None) applied here; ``out`` float32 [n, H vdim];
    ``state`` float32 [slots, H, dim, vdim]; the decays as float32 pairs hi + lo [H].  ``rotary`` = (cos, sin,
    rotated dimensions): q and k are rotated by position as they are read (dimension i paired with i + half; tables
    float32 [positions, half]); ``k_scale`` multiplies k behind the rotation."""
    _need(qkv, "qkv", contiguous=False); _need(out, "out", torch.float32); _need(state, "state", torch.float32)
    _need(decay_hi, "decay_hi", torch.float32); _need(decay_lo, "decay_lo", torch.float32)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    n = qkv.shape[0]
    if (tuple(out.shape) != (n, H * vdim) or tuple(state.shape[1:]) != (H, dim, vdim) or decay_hi.numel() != H
            or decay_lo.numel() != H or max(q_col, k_col) + H * dim > qkv.shape[1] or v_col + H * vdim > qkv.shape[1]):
        raise KernelError("lightning_scan: shape mismatch")
    if activation not in ("silu", None):
        raise KernelError("lightning_scan: activation is silu or none")
    if dim > LIGHTNING_MAX_DIM:
        raise KernelError(f"lightning_scan: dim={dim} exceeds {LIGHTNING_MAX_DIM}")
    cos, sin, rot = _lightning_rotary(rotary, dim, "lightning_scan")
    _run("lightning_scan", load_library("lightning").kp_lightning_scan, _ptr(qkv), _rows_2d(qkv, "qkv"), int(q_col), int(k_col),
         int(v_col), _ptr(decay_hi), _ptr(decay_lo), _ptr(state), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(out),
         _rows_2d(out, "out"), int(n_seg), H, dim, vdim, 0 if activation == "silu" else 1, int(bool(write_state)),
         _ptr(cos), _ptr(sin), rot, ctypes.c_float(k_scale), dtype_code(qkv.dtype), STREAM, work=(4 * n * H * dim * vdim, 0))
    return out


def _lightning_rotary(rotary, dim: int, what: str):
    """(cos, sin, rotated dimensions) checked; (None, None, 0) for no rotation."""
    if rotary is None:
        return None, None, 0
    cos, sin, rot = rotary
    if cos is None or not rot:
        return None, None, 0
    _need(cos, "cos", torch.float32); _need(sin, "sin", torch.float32)
    rot = int(rot)
    if rot < 2 or rot % 2 or rot > dim or cos.dim() != 2 or cos.shape[1] != rot // 2 or sin.shape != cos.shape:
        raise KernelError(f"{what}: rotation of {rot} dimensions does not go with heads of {dim} and tables {tuple(cos.shape)}")
    return cos, sin, rot


LIGHTNING_CHUNK_MAX_DIM = 128    # key rows of a head that the chunked form holds in shared memory


def lightning_chunk_rows() -> int:
    """Rows of a chunk of :func:`lightning_chunks` (its decay table holds the powers 0 .. rows of every head's decay)."""
    return int(load_library("lightning").kp_lightning_chunk_rows())


def lightning_chunks(qkv: torch.Tensor, q_col: int, k_col: int, v_col: int, decay_pow: torch.Tensor, state: torch.Tensor,
                     cu_rows: torch.Tensor, seg_pos: torch.Tensor, seg_slot: torch.Tensor, chunk_seg: torch.Tensor,
                     chunk_row0: torch.Tensor, seg_chunk0: torch.Tensor, n_chunks: int, out: torch.Tensor, n_seg: int,
                     H: int, dim: int, vdim: int, activation: Optional[str] = "silu", write_state: bool = True,
                     rotary=None, k_scale: float = 1.0) -> torch.Tensor:
    """The recurrence of :func:`lightning_scan` for segments of many rows: chunks of rows as small matrix products
    (float32 on the CUDA cores), the chunks of all segments side by side: every chunk's own sum, a short serial pass
    over a segment's chunks for the states at their heads, every chunk's outputs.  ``decay_pow``: float32
    [H, rows + 1], the powers ``a_h^m`` (made in double).  Sums have another order than the scan's.  ``chunk_seg`` /
    ``chunk_row0`` [n_chunks]: a chunk's segment and first row (chunks of at most :func:`lightning_chunk_rows` rows,
    a segment's chunks in order); ``seg_chunk0`` [n_seg + 1]: the first chunk of every segment.  ``rotary`` and
    ``k_scale`` as in :func:`lightning_scan`."""
    _need(qkv, "qkv", contiguous=False); _need(out, "out", torch.float32); _need(state, "state", torch.float32)
    _need(decay_pow, "decay_pow", torch.float32)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot"), (chunk_seg, "chunk_seg"),
                  (chunk_row0, "chunk_row0"), (seg_chunk0, "seg_chunk0")):
        _need(t, nm, torch.int32)
    n = qkv.shape[0]
    if (tuple(out.shape) != (n, H * vdim) or tuple(state.shape[1:]) != (H, dim, vdim)
            or tuple(decay_pow.shape) != (H, lightning_chunk_rows() + 1) or chunk_seg.numel() < n_chunks
            or chunk_row0.numel() < n_chunks or seg_chunk0.numel() < n_seg + 1
            or max(q_col, k_col) + H * dim > qkv.shape[1] or v_col + H * vdim > qkv.shape[1]):
        raise KernelError("lightning_chunks: shape mismatch")
    if activation not in ("silu", None):
        raise KernelError("lightning_chunks: activation is silu or none")
    if dim > LIGHTNING_CHUNK_MAX_DIM:
        raise KernelError(f"lightning_chunks: dim={dim} exceeds {LIGHTNING_CHUNK_MAX_DIM}")
    cos, sin, rot = _lightning_rotary(rotary, dim, "lightning_chunks")
    scratch = torch.empty(n_chunks * H * dim * vdim, dtype=torch.float32, device=qkv.device)
    _run("lightning_chunks", load_library("lightning").kp_lightning_chunks, _ptr(qkv), _rows_2d(qkv, "qkv"), int(q_col),
         int(k_col), int(v_col), _ptr(decay_pow), _ptr(state), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(chunk_seg),
         _ptr(chunk_row0), _ptr(seg_chunk0), int(n_chunks), _ptr(scratch), _ptr(out), _rows_2d(out, "out"), int(n_seg), H, dim,
         vdim, 0 if activation == "silu" else 1, int(bool(write_state)), _ptr(cos), _ptr(sin), rot, ctypes.c_float(k_scale),
         dtype_code(qkv.dtype), STREAM, work=(4 * n * H * dim * vdim, 0))
    LAUNCHES[0] += 2
    return out


# ------------------------------------------------------------------ selective state space (mamba2)

SSM_MAX_STATE = 256        # rows of a head's state that the scan keeps in registers
SSM_CHUNK_MAX_STATE = 128  # rows of a head's state that the chunked form holds in shared memory
SSM_MAX_TAPS = 16


def ssm_conv(p: torch.Tensor, conv_col: int, dt_col: int, taps: torch.Tensor, bias: torch.Tensor, dt_bias: torch.Tensor,
             a_log: torch.Tensor, kept: torch.Tensor, row_seg: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor,
             seg_slot: torch.Tensor, out: torch.Tensor, dt_out: torch.Tensor, da_out: torch.Tensor, n_seg: int,
             single_rows: bool, keep: bool = True) -> None:
    """``out = silu(conv(p[:, conv_col : conv_col + C]) + bias)`` (a causal convolution a channel, taps [C, K], the
    last tap on the current row; rows before a segment come from the request's kept inputs, zero at position 0),
    ``dt_out = softplus(p[:, dt_col : dt_col + H] + dt_bias)`` and ``da_out = -exp(a_log) * dt_out`` (float32).
    ``kept``: float32 [slots, stride] whose rows begin with the last K - 1 inputs as [K - 1, C]; renewed unless
    ``keep`` is False (``single_rows``: every segment has one row, and one launch does both)."""
    _need(p, "p", contiguous=False); _need(out, "out", p.dtype); _need(kept, "kept", torch.float32, contiguous=False)
    for t, nm in ((taps, "taps"), (bias, "bias"), (dt_bias, "dt_bias"), (a_log, "a_log"), (dt_out, "dt_out"), (da_out, "da_out")):
        _need(t, nm, torch.float32)
    for t, nm in ((row_seg, "row_seg"), (cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    n, C = out.shape
    H, K = dt_bias.numel(), taps.shape[1]
    if (p.shape[0] != n or tuple(taps.shape) != (C, K) or bias.numel() != C or a_log.numel() != H or tuple(dt_out.shape) != (n, H)
            or tuple(da_out.shape) != (n, H) or conv_col + C > p.shape[1] or dt_col + H > p.shape[1] or kept.dim() != 2
            or kept.stride(1) != 1 or kept.shape[1] < (K - 1) * C):
        raise KernelError("ssm_conv: shape mismatch")
    if K > SSM_MAX_TAPS:
        raise KernelError(f"ssm_conv: {K} taps exceed {SSM_MAX_TAPS}")
    _run("ssm_conv", load_library("ssm").kp_ssm_conv, _ptr(p), _rows_2d(p, "p"), int(conv_col), int(dt_col), _ptr(taps), _ptr(bias),
         _ptr(dt_bias), _ptr(a_log), _ptr(kept), ctypes.c_longlong(kept.stride(0)), _ptr(row_seg), _ptr(cu_rows), _ptr(seg_pos),
         _ptr(seg_slot), _ptr(out), _ptr(dt_out), _ptr(da_out), n, int(n_seg), C, H, K, int(bool(single_rows)), int(bool(keep)), 1,
         dtype_code(p.dtype), STREAM)
    if keep and not single_rows and K > 1:
        LAUNCHES[0] += 1


def channel_conv(p: torch.Tensor, conv_col: int, taps: torch.Tensor, kept: torch.Tensor, row_seg: torch.Tensor,
                 cu_rows: torch.Tensor, seg_pos: torch.Tensor, seg_slot: torch.Tensor, out: torch.Tensor, n_seg: int,
                 single_rows: bool, keep: bool = True, activation: Optional[str] = None,
                 bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """The convolution of :func:`ssm_conv` alone: ``out = act(conv(p[:, conv_col : conv_col + C]) (+ bias))``, act = silu
    or none.  ``kept`` as there."""
    _need(p, "p", contiguous=False); _need(out, "out", p.dtype); _need(kept, "kept", torch.float32, contiguous=False)
    _need(taps, "taps", torch.float32)
    for t, nm in ((row_seg, "row_seg"), (cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    n, C = out.shape
    K = taps.shape[1]
    if (p.shape[0] != n or tuple(taps.shape) != (C, K) or conv_col + C > p.shape[1] or kept.dim() != 2 or kept.stride(1) != 1
            or kept.shape[1] < (K - 1) * C):
        raise KernelError("channel_conv: shape mismatch")
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() != C:
            raise KernelError("channel_conv: bias size")
    if K > SSM_MAX_TAPS or activation not in ("silu", None):
        raise KernelError(f"channel_conv: {K} taps (at most {SSM_MAX_TAPS}), activation '{activation}' (silu or none)")
    none = _ptr(None)
    _run("channel_conv", load_library("ssm").kp_ssm_conv, _ptr(p), _rows_2d(p, "p"), int(conv_col), 0, _ptr(taps), _ptr(bias),
         none, none, _ptr(kept), ctypes.c_longlong(kept.stride(0)), _ptr(row_seg), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot),
         _ptr(out), none, none, n, int(n_seg), C, 0, K, int(bool(single_rows)), int(bool(keep)), int(activation == "silu"),
         dtype_code(p.dtype), STREAM)
    if keep and not single_rows and K > 1:
        LAUNCHES[0] += 1
    return out


def _ssm_check(what, xbc, dt, da, D, state, y, H, G, N, P):
    _need(xbc, "xbc", contiguous=False); _need(y, "y", torch.float32); _need(state, "state", torch.float32, contiguous=False)
    for t, nm in ((dt, "dt"), (da, "da"), (D, "D")):
        _need(t, nm, torch.float32)
    n = xbc.shape[0]
    if (tuple(y.shape) != (n, H * P) or tuple(dt.shape) != (n, H) or tuple(da.shape) != (n, H) or D.numel() != H or H % G
            or xbc.shape[1] < H * P + 2 * G * N or state.dim() != 2 or state.stride(1) != 1 or state.shape[1] < H * N * P):
        raise KernelError(f"{what}: shape mismatch")
    return n


def ssm_scan(xbc: torch.Tensor, dt: torch.Tensor, da: torch.Tensor, D: torch.Tensor, state: torch.Tensor, cu_rows: torch.Tensor,
             seg_pos: torch.Tensor, seg_slot: torch.Tensor, y: torch.Tensor, n_seg: int, H: int, G: int, N: int, P: int,
             write_state: bool = True) -> torch.Tensor:
    """``S <- exp(da) S + dt B x^T; y = S^T C + D x`` row after row of every segment, from the state in the segment's
    slot (zero at position 0) and back into it.  ``xbc`` rows hold [x: H heads of P | B: G groups of N | C: the same]
    in the storage type; ``dt``, ``da`` float32 [n, H]; ``state`` float32 [slots, stride] whose rows begin with
    [H, N, P]; ``y`` float32 [n, H P]."""
    n = _ssm_check("ssm_scan", xbc, dt, da, D, state, y, H, G, N, P)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    if N > SSM_MAX_STATE:
        raise KernelError(f"ssm_scan: state={N} exceeds {SSM_MAX_STATE}")
    _run("ssm_scan", load_library("ssm").kp_ssm_scan, _ptr(xbc), _rows_2d(xbc, "xbc"), H * P, H * P + G * N, _ptr(dt), _ptr(da),
         _ptr(D), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(y),
         _rows_2d(y, "y"), int(n_seg), H, G, N, P, int(bool(write_state)), dtype_code(xbc.dtype), STREAM,
         work=(4 * n * H * N * P, 0))
    return y


def ssm_chunk_rows() -> int:
    return int(load_library("ssm").kp_ssm_chunk_rows())


def ssm_chunks(xbc: torch.Tensor, dt: torch.Tensor, da: torch.Tensor, D: torch.Tensor, state: torch.Tensor, cu_rows: torch.Tensor,
               seg_pos: torch.Tensor, seg_slot: torch.Tensor, chunk_seg: torch.Tensor, chunk_row0: torch.Tensor,
               seg_chunk0: torch.Tensor, n_chunks: int, y: torch.Tensor, n_seg: int, H: int, G: int, N: int, P: int,
               write_state: bool = True) -> torch.Tensor:
    """The recurrence of :func:`ssm_scan` for segments of many rows, chunks of rows as small float32 matrix products,
    the chunks of all segments side by side (C B^T a group, sums, a serial pass over a segment's chunks, outputs).  The chunk lists
    as in :func:`lightning_chunks`.  Sums have another order than the scan's."""
    n = _ssm_check("ssm_chunks", xbc, dt, da, D, state, y, H, G, N, P)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot"), (chunk_seg, "chunk_seg"),
                  (chunk_row0, "chunk_row0"), (seg_chunk0, "seg_chunk0")):
        _need(t, nm, torch.int32)
    if chunk_seg.numel() < n_chunks or chunk_row0.numel() < n_chunks or seg_chunk0.numel() < n_seg + 1:
        raise KernelError("ssm_chunks: chunk lists too short")
    if N > SSM_CHUNK_MAX_STATE:
        raise KernelError(f"ssm_chunks: state={N} exceeds {SSM_CHUNK_MAX_STATE}")
    lib = load_library("ssm")
    lib.kp_ssm_chunks_scratch.restype = ctypes.c_longlong
    scratch = torch.empty(int(lib.kp_ssm_chunks_scratch(int(n_chunks), H, G, N, P)), dtype=torch.float32, device=xbc.device)
    _run("ssm_chunks", load_library("ssm").kp_ssm_chunks, _ptr(xbc), _rows_2d(xbc, "xbc"), H * P, H * P + G * N, _ptr(dt), _ptr(da),
         _ptr(D), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(chunk_seg),
         _ptr(chunk_row0), _ptr(seg_chunk0), int(n_chunks), _ptr(scratch), _ptr(y), _rows_2d(y, "y"), int(n_seg), H, G, N, P,
         int(bool(write_state)), dtype_code(xbc.dtype), STREAM, work=(4 * n * H * N * P, 0))
    LAUNCHES[0] += 3
    return y


# ------------------------------------------------------------------ recurrences with data-dependent decays

RECUR_MAX_DIM = 256        # key rows of a head's state
RECUR_MAX_TAPS = SSM_MAX_TAPS


def delta_prep(p: torch.Tensor, conv_col: int, b_col: int, a_col: int, taps: torch.Tensor, neg_a: torch.Tensor, dt_bias: torch.Tensor,
               kept: torch.Tensor, row_seg: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor, seg_slot: torch.Tensor,
               out: torch.Tensor, beta: torch.Tensor, lg: torch.Tensor, n_seg: int, H: int, G: int, D: int, P: int, q_scale: float,
               per_channel: bool, single_rows: bool, keep: bool = True) -> None:
    """What stands between the projections ``p`` and a delta recurrence.  ``out`` float32 [n, C]: the C = 2 G D + H P
    channels [q | k | v] from ``conv_col``, each behind its causal convolution (taps [C, K], the last on the current
    row) and silu, q and k as unit vectors a head, q times ``q_scale``.  ``beta`` [n, H] = sigmoid of the H columns from
    ``b_col``.  ``lg``: the logarithms of the decays, ``neg_a_h * softplus(z + dt_bias)`` with ``neg_a`` = -exp(A_log): a head
    (z the H columns from ``a_col``; lg [n, H]) or, ``per_channel``, a key channel (lg [n, H D] holds z and is changed in place).
    ``kept`` and ``single_rows`` as in :func:`ssm_conv`."""
    _need(p, "p", contiguous=False); _need(kept, "kept", torch.float32, contiguous=False)
    for t, nm in ((taps, "taps"), (neg_a, "neg_a"), (dt_bias, "dt_bias"), (out, "out"), (beta, "beta"), (lg, "lg")):
        _need(t, nm, torch.float32)
    for t, nm in ((row_seg, "row_seg"), (cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    n, C, K = p.shape[0], 2 * G * D + H * P, taps.shape[1]
    n_dec = H * D if per_channel else H
    if (tuple(out.shape) != (n, C) or tuple(taps.shape) != (C, K) or neg_a.numel() != H or dt_bias.numel() != n_dec
            or tuple(beta.shape) != (n, H) or tuple(lg.shape) != (n, n_dec) or conv_col + C > p.shape[1] or b_col + H > p.shape[1]
            or (not per_channel and a_col + H > p.shape[1]) or kept.dim() != 2 or kept.stride(1) != 1 or kept.shape[1] < (K - 1) * C):
        raise KernelError("delta_prep: shape mismatch")
    if K > RECUR_MAX_TAPS or D > RECUR_MAX_DIM:
        raise KernelError(f"delta_prep: {K} taps or heads of {D} exceed {RECUR_MAX_TAPS} or {RECUR_MAX_DIM}")
    _run("delta_prep", load_library("recurrence").kp_delta_prep, _ptr(p), _rows_2d(p, "p"), int(conv_col), int(b_col), int(a_col), _ptr(taps),
         _ptr(neg_a), _ptr(dt_bias), _ptr(kept), ctypes.c_longlong(kept.stride(0)), _ptr(row_seg), _ptr(cu_rows), _ptr(seg_pos),
         _ptr(seg_slot), _ptr(out), _ptr(beta), _ptr(lg), n, int(n_seg), H, G, D, P, K, ctypes.c_float(q_scale), int(bool(per_channel)),
         int(bool(single_rows)), int(bool(keep)), dtype_code(p.dtype), STREAM, work=(0, n * C * (p.element_size() + 4)))
    if keep and not single_rows and K > 1:
        LAUNCHES[0] += 1


def log_decay_sigmoid(z: torch.Tensor, tau: float) -> torch.Tensor:
    """z <- log(sigmoid(z)^(1 / tau)), in place, float32."""
    _need(z, "z", torch.float32)
    _run("log_decay_sigmoid", load_library("recurrence").kp_log_decay_sigmoid, _ptr(z), ctypes.c_longlong(z.numel()),
         ctypes.c_float(1.0 / float(tau)), STREAM, work=(0, 8 * z.numel()))
    return z


def _recur_check(what, q, k, v, lg, beta, state, out, H, G, D, P, per_channel):
    for t, nm in ((q, "q"), (k, "k"), (v, "v")):
        _need(t, nm, q.dtype, contiguous=False)
    _need(lg, "lg", torch.float32); _need(out, "out", torch.float32); _need(state, "state", torch.float32, contiguous=False)
    n = q.shape[0]
    if (q.stride(0) != k.stride(0) or q.stride(0) != v.stride(0) or tuple(q.shape) != (n, G * D) or tuple(k.shape) != (n, G * D)
            or tuple(v.shape) != (n, H * P) or H % G or tuple(lg.shape) != (n, H * D if per_channel else H)
            or tuple(out.shape) != (n, H * P) or state.dim() != 2 or state.stride(1) != 1 or state.shape[1] < H * D * P):
        raise KernelError(f"{what}: shape mismatch")
    if beta is not None:
        _need(beta, "beta", torch.float32)
        if tuple(beta.shape) != (n, H):
            raise KernelError(f"{what}: beta's shape")
        if q.dtype != torch.float32:
            raise KernelError(f"{what}: the delta recurrence reads float32 vectors (what delta_prep leaves)")
    elif not per_channel:
        raise KernelError(f"{what}: the gated recurrence has one decay a key channel")
    if D > RECUR_MAX_DIM:
        raise KernelError(f"{what}: heads of {D} exceed {RECUR_MAX_DIM}")
    return n


def recur_scan(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, lg: torch.Tensor, beta: Optional[torch.Tensor], q_scale: float,
               state: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor, seg_slot: torch.Tensor, out: torch.Tensor,
               n_seg: int, H: int, G: int, D: int, P: int, per_channel: bool, write_state: bool = True) -> torch.Tensor:
    """``F = exp(lg) S; e = beta (v - F^T k)``, or v without ``beta``; ``S = F + k e^T; o = S^T (q_scale q)`` row after row of
    every segment, from the state in the segment's slot (zero at position 0) and back into it.  ``q``, ``k`` [n, G D] and ``v``
    [n, H P] are columns of rows of one pitch; ``lg`` float32 [n, H], or with ``per_channel`` [n, H D]; ``state``
    float32 [slots, stride] whose rows begin with [H, D, P]; ``out`` float32 [n, H P]."""
    n = _recur_check("recur_scan", q, k, v, lg, beta, state, out, H, G, D, P, per_channel)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot")):
        _need(t, nm, torch.int32)
    _run("recur_scan", load_library("recurrence").kp_recur_scan, _ptr(q), _ptr(k), _ptr(v), q.stride(0), _ptr(lg), _ptr(beta),
         ctypes.c_float(q_scale), _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(out),
         _rows_2d(out, "out"), int(n_seg), H, G, D, P, int(bool(per_channel)), int(bool(write_state)), dtype_code(q.dtype), STREAM,
         tag=f" {'delta' if beta is not None else 'gated'}", work=((6 if beta is not None else 4) * n * H * D * P, 8 * n_seg * H * D * P))
    return out


def recur_chunk_rows() -> int:
    return int(load_library("recurrence").kp_recur_chunk_rows())


RECUR_CHUNK_MAX_DIM = 128        # key rows and value columns of a head that the chunked form takes
RECUR_CHUNK_MAX_VALUE = 256


def recur_chunks_ok(D: int, P: int) -> bool:
    return D <= RECUR_CHUNK_MAX_DIM and P <= RECUR_CHUNK_MAX_VALUE


def recur_chunks(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, lg: torch.Tensor, beta: Optional[torch.Tensor], q_scale: float,
                 state: torch.Tensor, cu_rows: torch.Tensor, seg_pos: torch.Tensor, seg_slot: torch.Tensor, chunk_seg: torch.Tensor,
                 chunk_row0: torch.Tensor, seg_chunk0: torch.Tensor, n_chunks: int, out: torch.Tensor, n_seg: int, H: int, G: int,
                 D: int, P: int, per_channel: bool, write_state: bool = True) -> torch.Tensor:
    """The recurrence of :func:`recur_scan` for segments of many rows: chunks of rows as small matrix products (tensor
    cores, tf32 with both operands in two parts), in three passes (see csrc/recurrence.cu).  The chunk lists as in
    :func:`lightning_chunks`.  Sums have another order than the scan's."""
    n = _recur_check("recur_chunks", q, k, v, lg, beta, state, out, H, G, D, P, per_channel)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (seg_slot, "seg_slot"), (chunk_seg, "chunk_seg"),
                  (chunk_row0, "chunk_row0"), (seg_chunk0, "seg_chunk0")):
        _need(t, nm, torch.int32)
    if chunk_seg.numel() < n_chunks or chunk_row0.numel() < n_chunks or seg_chunk0.numel() < n_seg + 1:
        raise KernelError("recur_chunks: chunk lists too short")
    if not recur_chunks_ok(D, P):
        raise KernelError(f"recur_chunks: heads of {D} x {P} exceed {RECUR_CHUNK_MAX_DIM} x {RECUR_CHUNK_MAX_VALUE}")
    lib = load_library("recurrence")
    lib.kp_recur_chunks_scratch.restype = ctypes.c_longlong
    scratch = torch.empty(int(lib.kp_recur_chunks_scratch(int(n_chunks), H, D, P, int(beta is not None))), dtype=torch.float32,
                          device=q.device)
    _run("recur_chunks", lib.kp_recur_chunks, _ptr(q), _ptr(k), _ptr(v), q.stride(0), _ptr(lg), _ptr(beta), ctypes.c_float(q_scale),
         _ptr(state), ctypes.c_longlong(state.stride(0)), _ptr(cu_rows), _ptr(seg_pos), _ptr(seg_slot), _ptr(chunk_seg), _ptr(chunk_row0),
         _ptr(seg_chunk0), int(n_chunks), _ptr(scratch), _ptr(out), _rows_2d(out, "out"), int(n_seg), H, G, D, P, int(bool(per_channel)),
         int(bool(write_state)), dtype_code(q.dtype), STREAM, tag=f" {'delta' if beta is not None else 'gated'}",
         work=((6 if beta is not None else 4) * n * H * D * P, 0))
    LAUNCHES[0] += 2
    return out


# ------------------------------------------------------------------ a residual of several streams

STREAMS_MAX = 8


def streams_enter(e: torch.Tensor, x: torch.Tensor) -> torch.Tensor:
    """x[r, s] = e[r] for every stream s: ``e`` float32 [n, d], ``x`` float32 [n, S, d]."""
    _need(e, "e", torch.float32); _need(x, "x", torch.float32)
    n, S, d = x.shape
    if tuple(e.shape) != (n, d):
        raise KernelError("streams_enter: shape mismatch")
    _run("streams_enter", load_library("streams").kp_streams_enter, _ptr(e), _ptr(x), n, d, S, STREAM)
    return x


def streams_rows(x: torch.Tensor, y: Optional[torch.Tensor] = None, mix: Optional[torch.Tensor] = None,
                 out_w: Optional[torch.Tensor] = None, in_w: Optional[torch.Tensor] = None, norm_w: Optional[torch.Tensor] = None,
                 eps: float = 0.0, centred: bool = True, h: Optional[torch.Tensor] = None,
                 rows: Optional[torch.Tensor] = None) -> None:
    """One pass over rows of several streams, ``x`` float32 [n, S, d].  With ``y`` (float32 [n, d], left cleared):
    ``x'_b = out_w_b y + sum_a mix_ab x_a``.  With ``h`` ([rows, d] in the storage type): ``h = norm(sum_t in_w[t] x_t) *
    norm_w`` of the new streams (``in_w`` None: their sum), the norm centred (a layer norm without a shift) or the RMS
    norm.  ``rows`` (without ``y``): the rows to read."""
    _need(x, "x", torch.float32)
    n, S, d = x.shape
    if S > STREAMS_MAX:
        raise KernelError(f"streams_rows: {S} streams exceed {STREAMS_MAX}")
    if y is not None:
        for t, nm, size in ((y, "y", n * d), (mix, "mix", S * S), (out_w, "out_w", S)):
            _need(t, nm, torch.float32)
            if t.numel() != size:
                raise KernelError(f"streams_rows: size of {nm}")
        if rows is not None:
            raise KernelError("streams_rows: picked rows are read, not changed")
    if h is not None:
        _need(h, "h"); _need(norm_w, "norm_w", torch.float32)
        if rows is not None:
            _need(rows, "rows", torch.int32)
        n_out = n if rows is None else rows.numel()
        if tuple(h.shape) != (n_out, d) or norm_w.numel() != d:
            raise KernelError("streams_rows: shape mismatch")
        if in_w is not None:
            _need(in_w, "in_w", torch.float32)
            if in_w.numel() != S:
                raise KernelError("streams_rows: size of in_w")
    elif y is None or rows is not None:
        raise KernelError("streams_rows: nothing to do")
    n_rows = n if rows is None else rows.numel()
    if n_rows > MAX_STEP_ROWS:
        raise KernelError("streams_rows: too many rows")
    _run("streams_rows", load_library("streams").kp_streams_rows, _ptr(x), _ptr(y), _ptr(mix), _ptr(out_w), _ptr(in_w), _ptr(norm_w),
         ctypes.c_float(eps), int(bool(centred)), _ptr(rows), _ptr(h), n_rows, d, S, dtype_code(h.dtype if h is not None else torch.float32),
         STREAM, work=(0, n_rows * d * (4 * S * (2 if y is not None else 1) + (8 if y is not None else 0)
                                        + (h.element_size() if h is not None else 0))))


# ------------------------------------------------------------------ attention

def qk_norm_rope_kv(qkv: torch.Tensor, q_w: Optional[torch.Tensor], k_w: Optional[torch.Tensor], eps: float,
                    cos_tab: Optional[torch.Tensor], sin_tab: Optional[torch.Tensor], rotary_dim: int,
                    interleaved: bool, positions: torch.Tensor, slot_map: Optional[torch.Tensor],
                    q_out: Optional[torch.Tensor], cache: Optional[torch.Tensor], page_size: int, H: int, G: int,
                    hd: int, v_col: Optional[int] = None, norm_dim: Optional[int] = None,
                    q_temp: Optional[Tuple[float, float]] = None, norm_after: bool = False) -> Optional[torch.Tensor]:
    """Norm + rotate q and k; write q to ``q_out`` and, if ``cache`` is given,
    k and v to their pages.  ``cache`` is one layer's [pages, 2, G, page_size, hd].
    With ``q_out`` None, q and k are changed in place and no cache is written.
    ``v_col``: the column of a row at which the values start (default: behind the keys, ``(H + G) * hd``;
    ``H * hd`` makes the values the key projections themselves, before norm and rotation).  Columns behind
    q, k and v are left alone.  ``norm_dim``: the number the norm's mean is taken over where a head is stored
    wider than it is (zeros behind its own columns; default ``hd``).  ``q_temp`` = (coef, every): the queries of
    the row at position p leave multiplied by ``1 + coef ln(floor((p + 1) / every) + 1)`` (float32).  ``norm_after``: q
    and k are divided by their root mean square (``eps``, no weight) behind the rotation, not in front of it."""
    _need(qkv, "qkv", contiguous=False)
    _need(positions, "positions", torch.int32)
    n = qkv.shape[0]
    if v_col is None:
        v_col = (H + G) * hd
    if qkv.shape[1] < (H + G) * hd or not (0 <= v_col <= qkv.shape[1] - G * hd):
        raise KernelError("qk_norm_rope_kv: shape mismatch")
    if q_out is None and v_col < (H + G) * hd:
        raise KernelError("qk_norm_rope_kv: the in-place form would change the values it shares with the keys")
    if q_out is not None:
        _need(q_out, "q_out", qkv.dtype, contiguous=False)
        if q_out.shape != (n, H * hd):
            raise KernelError("qk_norm_rope_kv: q_out shape")
    elif cache is not None:
        raise KernelError("qk_norm_rope_kv: the in-place form writes no cache")
    for t, nm in ((q_w, "q_w"), (k_w, "k_w")):
        if t is not None:
            _need(t, nm, torch.float32)
            if t.numel() != hd:
                raise KernelError(f"qk_norm_rope_kv: {nm} size")
    if cos_tab is not None:
        _need(cos_tab, "cos_tab", torch.float32); _need(sin_tab, "sin_tab", torch.float32)
        if cos_tab.shape[1] != rotary_dim // 2:
            raise KernelError("qk_norm_rope_kv: table width")
    write_kv = cache is not None
    if write_kv:
        _need(cache, "cache", qkv.dtype); _need(slot_map, "slot_map", torch.int32)
        if tuple(cache.shape[1:]) != (2, G, page_size, hd):
            raise KernelError(f"qk_norm_rope_kv: cache layout {tuple(cache.shape)}")
    nd = hd if norm_dim is None else int(norm_dim)
    if not (1 <= nd <= hd):
        raise KernelError("qk_norm_rope_kv: norm_dim")
    if norm_after and (q_w is not None or k_w is not None or q_out is None):
        raise KernelError("qk_norm_rope_kv: the norm behind the rotation has no weights and no in-place form")
    coef, every = (0.0, 0.0) if q_temp is None else (float(q_temp[0]), float(q_temp[1]))
    if q_temp is not None and not every > 0:
        raise KernelError("qk_norm_rope_kv: the query temperature's period must be positive")
    lib = load_library("qkrope")
    _run("qk_norm_rope_kv", lib.kp_qk_norm_rope_kv_after, _ptr(qkv), _rows_2d(qkv, "qkv"), _ptr(q_w), _ptr(k_w), ctypes.c_float(eps),
                                  _ptr(cos_tab), _ptr(sin_tab), rotary_dim, int(interleaved), _ptr(positions),
                                  _ptr(slot_map), _ptr(q_out), 0 if q_out is None else _rows_2d(q_out, "q_out"), _ptr(cache),
                                  page_size,
                                  n, H, G, hd, int(write_kv), int(v_col), nd, ctypes.c_float(coef), ctypes.c_float(every),
                                  int(bool(norm_after)), dtype_code(qkv.dtype), STREAM)
    return q_out


def qk_rownorm_kv(qkv: torch.Tensor, k_col: int, v_col: int, q_w: torch.Tensor, k_w: Optional[torch.Tensor], eps: float,
                  count_q: int, count_k: int, slot_map: Optional[torch.Tensor], q_out: torch.Tensor,
                  cache: Optional[torch.Tensor], page_size: int, H: int, G: int, hd: int) -> torch.Tensor:
    """RMS norm of q and of k each over its whole projection (all heads at once, weights as long as the projections),
    no rotation; q to ``q_out``, and with ``cache`` given the normed k and v to their pages.  Rows hold q at column
    0 (H heads stored ``hd`` wide), k at ``k_col`` and v at ``v_col`` (G heads each).  ``count_q`` / ``count_k``: the
    numbers the means are taken over (smaller than H hd and G hd where heads are stored wider than they are, with
    zeros behind)."""
    _need(qkv, "qkv", contiguous=False); _need(q_out, "q_out", qkv.dtype); _need(q_w, "q_w", torch.float32)
    n = qkv.shape[0]
    if tuple(q_out.shape) != (n, H * hd) or q_w.numel() != H * hd or H * hd > qkv.shape[1]:
        raise KernelError("qk_rownorm_kv: shape mismatch")
    write_kv = cache is not None
    if write_kv:
        _need(cache, "cache", qkv.dtype); _need(slot_map, "slot_map", torch.int32); _need(k_w, "k_w", torch.float32)
        if (tuple(cache.shape[1:]) != (2, G, page_size, hd) or k_w.numel() != G * hd
                or max(k_col, v_col) + G * hd > qkv.shape[1] or min(k_col, v_col) < H * hd):
            raise KernelError(f"qk_rownorm_kv: cache layout {tuple(cache.shape)} or columns")
    if n > MAX_STEP_ROWS:
        raise KernelError("qk_rownorm_kv: too many rows")
    _run("qk_rownorm_kv", load_library("qkrope").kp_qk_rownorm_kv, _ptr(qkv), _rows_2d(qkv, "qkv"), int(k_col), int(v_col),
         _ptr(q_w), _ptr(k_w if write_kv else None), ctypes.c_float(eps), ctypes.c_float(count_q), ctypes.c_float(count_k),
         _ptr(slot_map if write_kv else None), _ptr(q_out), H * hd, _ptr(cache), page_size, n, H, G, hd, int(write_kv),
         dtype_code(qkv.dtype), STREAM)
    return q_out


def pool_blocks(cache: torch.Tensor, block_table: torch.Tensor, row_seg: torch.Tensor, positions: torch.Tensor,
                pool_slot_map: torch.Tensor, pool_cache: torch.Tensor, pool: int, page_size: int, G: int, hd: int) -> None:
    """The means of the blocks of ``pool`` positions that this step's rows complete, from the keys and values in ``cache``
    (this step's already in it) to the entries ``pool_slot_map`` names (-1: the row completes no block)."""
    _need(cache, "cache"); _need(pool_cache, "pool_cache", cache.dtype)
    for t, nm in ((block_table, "block_table"), (row_seg, "row_seg"), (positions, "positions"), (pool_slot_map, "pool_slot_map")):
        _need(t, nm, torch.int32)
    n = positions.numel()
    for c in (cache, pool_cache):
        if tuple(c.shape[1:]) != (2, G, page_size, hd):
            raise KernelError(f"pool_blocks: cache layout {tuple(c.shape)}")
    if row_seg.numel() != n or pool_slot_map.numel() != n or pool < 1:
        raise KernelError("pool_blocks: shape mismatch")
    _run("pool_blocks", load_library("qkrope").kp_pool_blocks, _ptr(cache), _ptr(block_table), block_table.shape[1], _ptr(row_seg),
         _ptr(positions), _ptr(pool_slot_map), _ptr(pool_cache), int(pool), page_size, n, G, hd, dtype_code(cache.dtype), STREAM)


class Pooled:
    """What the attention kernels need to read the means of blocks of positions behind a window: the positions a block
    (``pool``), the layer's cache of the means and the requests' block tables into it."""

    def __init__(self, pool: int, cache: torch.Tensor, block_table: torch.Tensor):
        self.pool, self.cache, self.block_table = int(pool), cache, block_table

    def check(self, cache: torch.Tensor, window, keep_first, block, what: str) -> None:
        _need(self.cache, "pooled cache", cache.dtype); _need(self.block_table, "pooled block table", torch.int32)
        if self.pool < 1 or not window or keep_first or block:
            raise KernelError(f"{what}: pooled blocks go with a window, and not with kept first keys or blocks of positions")
        if self.cache.shape[1:] != cache.shape[1:]:
            raise KernelError(f"{what}: the pooled cache is laid out like the cache")

    def chunks(self, n_chunks: int) -> int:
        """Chunks of SPLIT_CHUNK entries that a context of ``n_chunks`` chunks of keys can have."""
        return -(-(n_chunks * SPLIT_CHUNK // self.pool) // SPLIT_CHUNK) or 1


def _pool_args(pooled: Optional[Pooled]):
    if pooled is None:
        return 0, _ptr(None), _ptr(None), 0
    return pooled.pool, _ptr(pooled.cache), _ptr(pooled.block_table), pooled.block_table.shape[1]


def _check_sink(sink: Optional[torch.Tensor], H: int, keep_first: int, window: Optional[int], block: Optional[int], what: str) -> None:
    if sink is not None:
        _need(sink, "sink", torch.float32)
        if sink.numel() != H:
            raise KernelError(f"{what}: one sink a query head")
    if keep_first and (keep_first < 0 or block):
        raise KernelError(f"{what}: keep_first must not be negative and does not go with blocks of positions")


def attention_rows(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, row_seg: torch.Tensor,
                   positions: torch.Tensor, out: torch.Tensor, scale: float, window: Optional[int],
                   page_size: int, H: int, G: int, hd: int, block: Optional[int] = None, keep_first: int = 0,
                   sink: Optional[torch.Tensor] = None, cap: float = 0.0, out_scale: float = 1.0,
                   pooled: Optional[Pooled] = None) -> torch.Tensor:
    """``block``: a row reads no key from before the start of its own block of that many positions.
    ``keep_first``: behind its window a row still reads the first that many keys of its sequence.  ``sink``
    (float32 [H]): ``exp(sink_h)`` joins the softmax's denominator, a key with a score and no value.  ``cap`` (0: none)
    bounds the scores, ``cap tanh(s / cap)``; ``out_scale`` multiplies the output; ``pooled``: behind its window a row also
    reads the means of the blocks of positions that lie wholly before it."""
    _need(q, "q", contiguous=False); _need(cache, "cache", q.dtype); _need(out, "out", q.dtype, contiguous=False)
    _need(block_table, "block_table", torch.int32); _need(row_seg, "row_seg", torch.int32)
    _need(positions, "positions", torch.int32)
    n = q.shape[0]
    if q.shape[1] != H * hd or out.shape != (n, H * hd) or tuple(cache.shape[1:]) != (2, G, page_size, hd):
        raise KernelError("attention_rows: shape mismatch")
    _check_sink(sink, H, keep_first, window, block, "attention_rows")
    if pooled is not None:
        pooled.check(cache, window, keep_first, block, "attention_rows")
    lib = load_library("attention")
    _run("attention_rows", lib.kp_attention_rows_pooled, _ptr(q), _rows_2d(q, "q"), _ptr(cache), _ptr(block_table),
         block_table.shape[1], _ptr(row_seg), _ptr(positions), _ptr(out), _rows_2d(out, "out"), ctypes.c_float(scale),
         int(window or 0), int(block or 0), int(keep_first or 0), _ptr(sink), ctypes.c_float(cap), ctypes.c_float(out_scale),
         *_pool_args(pooled), page_size, n, H, G, hd, dtype_code(q.dtype), STREAM)
    return out


SPLIT_CHUNK = 256          # keys a chunk of the split-KV attention
SPLIT_CHUNK_MMA = 256       # keys a chunk of its tensor-core form: 64, 128 or 256 (a divisor of SPLIT_CHUNK)
SPLIT_MAX_RATIO = 8        # query heads per kv head it takes


def attention_split_scratch(n_rows: int, H: int, hd: int, n_chunks: int, keep_first: int = 0,
                            pooled: Optional["Pooled"] = None) -> int:
    """Float elements of scratch that :func:`attention_split` needs (``keep_first``: with slots for the chunks of
    that many kept first keys; ``pooled``: for those of the pooled entries)."""
    slots = n_chunks * (SPLIT_CHUNK // min(SPLIT_CHUNK, SPLIT_CHUNK_MMA)) + -(-int(keep_first or 0) // SPLIT_CHUNK)
    if pooled is not None:
        slots += pooled.chunks(n_chunks) * (SPLIT_CHUNK // min(SPLIT_CHUNK, SPLIT_CHUNK_MMA))
    return n_rows * H * slots * (hd + 2)


def attention_split(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, row_seg: torch.Tensor,
                    positions: torch.Tensor, out: torch.Tensor, scratch: torch.Tensor, n_chunks: int, scale: float,
                    window: Optional[int], page_size: int, H: int, G: int, hd: int,
                    block: Optional[int] = None, exact_weights: bool = False, keep_first: int = 0,
                    sink: Optional[torch.Tensor] = None, cap: float = 0.0, out_scale: float = 1.0,
                    pooled: Optional[Pooled] = None) -> torch.Tensor:
    """Split-KV attention (chunks of 256 keys, merged in order).  ``n_chunks``
    must cover the largest position of the batch; ``scratch`` is float32.
    ``block``: a row reads no key from before the start of its own block of that many positions.
    ``exact_weights``: the softmax weights enter the product with V whole (the scalar kernel always does so; the
    tensor-core form then multiplies their three bfloat16 parts one after the other) instead of rounded to bfloat16.
    ``keep_first`` / ``sink``: as in :func:`attention_rows`; the sink enters in the merge, once a row; kept first
    keys behind a window are computed by a second small launch where the tensor-core form (which knows nothing of
    them) computes the window's chunks.  ``cap``, ``out_scale``, ``pooled``: as there too; the pooled entries' chunks are
    computed by a launch of their own, the output's factor enters in the merge."""
    _need(q, "q", contiguous=False); _need(cache, "cache", q.dtype); _need(out, "out", q.dtype, contiguous=False)
    _need(block_table, "block_table", torch.int32); _need(row_seg, "row_seg", torch.int32)
    _need(positions, "positions", torch.int32); _need(scratch, "scratch", torch.float32)
    n = q.shape[0]
    if q.shape[1] != H * hd or out.shape != (n, H * hd) or tuple(cache.shape[1:]) != (2, G, page_size, hd):
        raise KernelError("attention_split: shape mismatch")
    keep_first = int(keep_first or 0) if window else 0
    if scratch.numel() < attention_split_scratch(n, H, hd, n_chunks, keep_first, pooled):
        raise KernelError("attention_split: scratch too small")
    _check_sink(sink, H, keep_first, window, block, "attention_split")
    if pooled is not None:
        pooled.check(cache, window, keep_first, block, "attention_split")
    lib = load_library("attention_decode")
    if USE_MMA_ATTENTION and q.dtype == torch.bfloat16 and hd in (64, 128) and q.stride(0) % 2 == 0:
        # tensor-core chunk pass over smaller chunks, then the same merge; kept first keys get slots behind the window's
        # chunks (for the chunk pass they are chunks beyond every position: it leaves them alone)
        front0 = n_chunks * (SPLIT_CHUNK // SPLIT_CHUNK_MMA)
        pool_chunks = pooled.chunks(n_chunks) * (SPLIT_CHUNK // SPLIT_CHUNK_MMA) if pooled is not None else 0
        parts = front0 + -(-keep_first // SPLIT_CHUNK) + pool_chunks
        if keep_first:
            _run("attention_front_chunks", lib.kp_attention_front_chunks, _ptr(q), _rows_2d(q, "q"), _ptr(cache), _ptr(block_table),
                 block_table.shape[1], _ptr(row_seg), _ptr(positions), _ptr(scratch), parts, front0, ctypes.c_float(scale),
                 int(window), keep_first, page_size, n, H, G, hd, dtype_code(q.dtype), STREAM)
        mma = load_library("attention_mma").kp_attention_split_mma_pooled
        _run("attention_split_mma", mma,
            _ptr(q), _rows_2d(q, "q"), _ptr(cache), ctypes.c_longlong(cache.shape[0] if USE_TMA_ATTENTION else 0),
            _ptr(block_table), block_table.shape[1], _ptr(row_seg),
            _ptr(positions), _ptr(scratch), front0, parts, 0, SPLIT_CHUNK_MMA, ctypes.c_float(scale), int(window or 0), int(block or 0),
            int(bool(exact_weights)), ctypes.c_float(cap), 0, page_size, n, H, G, hd, STREAM)
        if pooled is not None:
            _run("attention_split_pool", mma,
                _ptr(q), _rows_2d(q, "q"), _ptr(pooled.cache), ctypes.c_longlong(pooled.cache.shape[0] if USE_TMA_ATTENTION else 0),
                _ptr(pooled.block_table), pooled.block_table.shape[1], _ptr(row_seg),
                _ptr(positions), _ptr(scratch), pool_chunks, parts, front0, SPLIT_CHUNK_MMA, ctypes.c_float(scale), int(window), 0,
                int(bool(exact_weights)), ctypes.c_float(cap), pooled.pool, page_size, n, H, G, hd, STREAM)
        _run("attention_merge", lib.kp_attention_merge_pooled, _ptr(positions), _ptr(out), _rows_2d(out, "out"), _ptr(scratch),
             parts, SPLIT_CHUNK_MMA, int(window or 0), int(block or 0), keep_first, _ptr(sink),
             front0 if keep_first or pooled is not None else -1, ctypes.c_float(out_scale), pooled.pool if pooled is not None else 0,
             n, H, hd, dtype_code(q.dtype), STREAM)
        return out
    _run("attention_split", lib.kp_attention_split_pooled, _ptr(q), _rows_2d(q, "q"), _ptr(cache), _ptr(block_table),
         block_table.shape[1], _ptr(row_seg), _ptr(positions), _ptr(out), _rows_2d(out, "out"), _ptr(scratch),
         n_chunks, ctypes.c_float(scale), int(window or 0), int(block or 0), keep_first, _ptr(sink), ctypes.c_float(cap),
         ctypes.c_float(out_scale), *_pool_args(pooled), pooled.chunks(n_chunks) if pooled is not None else 0, page_size, n, H, G, hd,
         dtype_code(q.dtype), STREAM)
    LAUNCHES[0] += 1 if pooled is None else 2
    return out


USE_TMA_ATTENTION = True       # its key/value tiles come by TMA where the page size allows
USE_MMA_ATTENTION = True       # bfloat16 attention with head size 64 or 128 runs on the tensor cores
PREFILL_TILE = 64              # query rows a CTA of the prefill attention kernel


USE_TC_ATTENTION = True        # prompt portions with head size 64 run on the tcgen05 tensor cores


def attention_prefill_tc_ok(q: torch.Tensor, out: torch.Tensor, cache: torch.Tensor, page_size: int, hd: int) -> bool:
    """Can the tcgen05 prefill attention take this call (head size 64, 16-byte aligned rows, a page size
    that is a multiple of 8 and divides 128 or is a multiple of it)?"""
    return (USE_TC_ATTENTION and hd == 64 and q.stride(0) % 8 == 0 and out.stride(0) % 8 == 0
            and q.data_ptr() % 16 == 0 and out.data_ptr() % 16 == 0 and cache.data_ptr() % 16 == 0
            and page_size % 8 == 0 and (page_size % 128 == 0 or 128 % page_size == 0)
            and cache.shape[0] * cache.shape[1] * cache.shape[2] * page_size < 2 ** 31 - 1)


def attention_prefill_ok(q: torch.Tensor, hd: int) -> bool:
    return USE_MMA_ATTENTION and q.dtype == torch.bfloat16 and hd in (64, 128) and q.stride(0) % 2 == 0


def attention_prefill(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, cu_rows: torch.Tensor,
                      seg_pos: torch.Tensor, tile_seg: torch.Tensor, tile_row0: torch.Tensor, out: torch.Tensor,
                      scale: float, window: Optional[int], page_size: int, H: int, G: int, hd: int,
                      big_tile_seg: Optional[torch.Tensor] = None, big_tile_row0: Optional[torch.Tensor] = None,
                      block: Optional[int] = None, exact_weights: bool = False, keep_first: int = 0,
                      sink: Optional[torch.Tensor] = None, cap: float = 0.0, out_scale: float = 1.0,
                      pooled: Optional[Pooled] = None) -> torch.Tensor:
    """Tensor-core causal attention for segments of many rows.  ``tile_seg`` / ``tile_row0`` list, for every
    tile of 64 consecutive rows of a segment, its segment and its first row; ``big_tile_seg`` /
    ``big_tile_row0`` the same for tiles of 128 rows, the tile that reads the most keys first (with them the
    tcgen05 kernel runs where it takes the sizes).  ``block``: a row reads no key from before the start of its own
    block of that many positions.  ``exact_weights``: the softmax weights enter the product with V whole, as three
    bfloat16 parts multiplied one after the other (the mma.sync kernel; the tcgen05 kernel, whose weights pass
    through shared memory as one bfloat16 operand, is then not taken).  ``keep_first`` / ``sink`` / ``cap`` / ``out_scale`` /
    ``pooled``: as in :func:`attention_rows` (the mma.sync kernel has them, the tcgen05 kernel is then not taken)."""
    _need(q, "q", torch.bfloat16, contiguous=False); _need(cache, "cache", torch.bfloat16)
    _need(out, "out", torch.bfloat16, contiguous=False)
    for t_, nm in ((block_table, "block_table"), (cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (tile_seg, "tile_seg"),
                   (tile_row0, "tile_row0")):
        _need(t_, nm, torch.int32)
    n = q.shape[0]
    if q.shape[1] != H * hd or out.shape != (n, H * hd) or tuple(cache.shape[1:]) != (2, G, page_size, hd):
        raise KernelError("attention_prefill: shape mismatch")
    if tile_seg.numel() != tile_row0.numel():
        raise KernelError("attention_prefill: tile lists differ in length")
    _check_sink(sink, H, keep_first, window, block, "attention_prefill")
    if pooled is not None:
        pooled.check(cache, window, keep_first, block, "attention_prefill")
    keep_first = int(keep_first or 0) if window else 0
    if (big_tile_seg is not None and not exact_weights and not keep_first and sink is None and not cap and out_scale == 1.0
            and pooled is None and attention_prefill_tc_ok(q, out, cache, page_size, hd)):
        _need(big_tile_seg, "big_tile_seg", torch.int32); _need(big_tile_row0, "big_tile_row0", torch.int32)
        if big_tile_seg.numel() != big_tile_row0.numel():
            raise KernelError("attention_prefill: tile lists differ in length")
        _run("attention_prefill_tc", load_library("attention_tc").kp_attention_prefill_tc_masked,
            _ptr(q), _rows_2d(q, "q"), n, _ptr(cache), ctypes.c_longlong(cache.shape[0]), _ptr(block_table),
            block_table.shape[1], _ptr(cu_rows), _ptr(seg_pos), _ptr(big_tile_seg), _ptr(big_tile_row0),
            big_tile_seg.numel(),
            _ptr(out), _rows_2d(out, "out"), ctypes.c_float(scale), int(window or 0), int(block or 0), page_size, H, G, hd,
            STREAM)
        return out
    _run("attention_prefill_mma", load_library("attention_mma").kp_attention_prefill_mma_pooled,
        _ptr(q), _rows_2d(q, "q"), _ptr(cache), _ptr(block_table), block_table.shape[1], _ptr(cu_rows), _ptr(seg_pos),
        _ptr(tile_seg), _ptr(tile_row0), tile_seg.numel(), _ptr(out), _rows_2d(out, "out"), ctypes.c_float(scale),
        int(window or 0), int(block or 0), keep_first, _ptr(sink), int(bool(exact_weights)), ctypes.c_float(cap),
        ctypes.c_float(out_scale), *_pool_args(pooled), page_size, H, G, hd, STREAM)
    return out


# ------------------------------------------------------------------ attention over cached latents

LATENT_PREFILL_MAX = (256, 256)    # key and value columns a head that the expanded pass takes
USE_TC_LATENT = True           # both latent passes of bfloat16 rows run on the tcgen05 tensor cores where the sizes allow it


def latent_prep(p: torch.Tensor, q_col: int, c_col: int, H: int, dimp: int, rotp: int, rank: int, rankp: int, W: int, w: torch.Tensor,
                eps: float, rotary, positions: torch.Tensor, slot_map: torch.Tensor, cache: Optional[torch.Tensor],
                page_size: int, qa: Optional[torch.Tensor], n_absorbed: int) -> None:
    """Rows ``p`` of the input product hold H query heads of (dimp | rotp) at ``q_col`` and the latent (rankp) with the
    shared key part (rotp) at ``c_col``: norm the latent over its ``rank`` columns (weight ``w`` [rank]), rotate the key part
    and store both in the row's cache page; rotate the heads' query parts in place, and copy those of the first
    ``n_absorbed`` rows behind the absorbed queries in ``qa`` [n_absorbed, H, W].  A cache row and an absorbed query have ``W``
    elements, zeros behind their rankp + rotp.  ``rotary``: (cos, sin,
    dimensions, interleaved) as a position part gives it."""
    _need(p, "p", contiguous=False); _need(w, "w", torch.float32); _need(positions, "positions", torch.int32)
    n = p.shape[0]
    if (p.stride(1) != 1 or q_col + H * (dimp + rotp) > p.shape[1] or c_col + rankp + rotp > p.shape[1] or w.numel() != rank
            or W < rankp + rotp):
        raise KernelError("latent_prep: shape mismatch")
    if cache is not None:
        _need(cache, "cache", p.dtype); _need(slot_map, "slot_map", torch.int32)
        if tuple(cache.shape[1:]) != (1, 1, page_size, W):
            raise KernelError(f"latent_prep: cache layout {tuple(cache.shape)}")
    if n_absorbed:
        _need(qa, "qa", p.dtype)
        if tuple(qa.shape) != (n_absorbed, H, W):
            raise KernelError("latent_prep: qa shape")
    cos, sin, rot, inter = rotary
    if cos is not None:
        _need(cos, "cos", torch.float32); _need(sin, "sin", torch.float32)
        if cos.shape[1] != rot // 2 or rot > rotp:
            raise KernelError("latent_prep: table width")
    _run("latent_prep", load_library("latent").kp_latent_prep, _ptr(p), p.stride(0), int(q_col), int(c_col), H, dimp, rotp, rank, rankp,
         int(W), _ptr(w), ctypes.c_float(eps), _ptr(cos), _ptr(sin), int(rot), int(bool(inter)), _ptr(positions), _ptr(slot_map), _ptr(cache),
         page_size, _ptr(qa), int(n_absorbed), n, dtype_code(p.dtype), STREAM)


def head_gemm(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out[m, h, :] = a[m, h, :] @ b[h].T, times ``sigmoid(gate[m, h, :])`` if given.  ``a`` [M, H, K], ``out`` and ``gate``
    [M, H, N] may be strided views (last dimension dense); ``b`` [H, N, K]."""
    M, H, K = a.shape
    N = b.shape[1]
    _need(a, "a", contiguous=False); _need(b, "b", a.dtype); _need(out, "out", a.dtype, contiguous=False)
    if tuple(b.shape) != (H, N, K) or tuple(out.shape) != (M, H, N) or a.stride(2) != 1 or out.stride(2) != 1:
        raise KernelError(f"head_gemm: shapes a{tuple(a.shape)} b{tuple(b.shape)} out{tuple(out.shape)}")
    if gate is not None:
        _need(gate, "gate", a.dtype, contiguous=False)
        if tuple(gate.shape) != (M, H, N) or gate.stride(2) != 1:
            raise KernelError("head_gemm: gate shape")
    ll = ctypes.c_longlong
    _run("head_gemm", load_library("latent").kp_head_gemm, _ptr(a), ll(a.stride(0)), a.stride(1), _ptr(b), _ptr(out), ll(out.stride(0)),
         out.stride(1), _ptr(gate), ll(gate.stride(0) if gate is not None else 0), gate.stride(1) if gate is not None else 0, M, N, K, H,
         dtype_code(a.dtype), STREAM, tag=f" {H}x{N}x{K}", work=(2 * M * H * N * K, (H * N * K + M * H * (N + K)) * a.element_size()))
    return out


def latent_chunks(n: int, max_context: int, H: int, rankp: int, W: int, page_size: int, dtype: torch.dtype) -> int:
    """Chunks that :func:`latent_split` cuts a context of ``max_context`` keys into at most, for these sizes and ``n`` rows."""
    return int(load_library("latent").kp_latent_chunks(int(n), int(max_context), rankp, W, H, page_size, dtype_code(dtype), int(USE_TC_LATENT)))


def latent_split_scratch(n: int, H: int, rankp: int, W: int, max_context: int, page_size: int, dtype: torch.dtype) -> int:
    """Float elements of scratch that :func:`latent_split` needs."""
    return n * H * latent_chunks(n, max_context, H, rankp, W, page_size, dtype) * (rankp + 2)


def latent_split(qa: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, row_seg: torch.Tensor, positions: torch.Tensor,
                 scratch: torch.Tensor, max_context: int, u: torch.Tensor, scale: float, page_size: int) -> torch.Tensor:
    """Causal softmax attention of absorbed queries ``qa`` [n, H, W] over the cached rows (the latents are the values too):
    ``u`` [n, H, rankp].  ``max_context`` lies beyond the largest position; ``scratch`` is float32.  bfloat16 rows run
    on the tcgen05 tensor cores where the sizes allow it."""
    n, H, W = qa.shape
    rankp = u.shape[2]
    _need(qa, "qa"); _need(cache, "cache", qa.dtype); _need(u, "u", qa.dtype); _need(scratch, "scratch", torch.float32)
    for t, nm in ((block_table, "block_table"), (row_seg, "row_seg"), (positions, "positions")):
        _need(t, nm, torch.int32)
    if tuple(cache.shape[1:]) != (1, 1, page_size, W) or tuple(u.shape) != (n, H, rankp) or row_seg.numel() != n or positions.numel() != n:
        raise KernelError("latent_split: shape mismatch")
    if scratch.numel() < latent_split_scratch(n, H, rankp, W, max_context, page_size, qa.dtype):
        raise KernelError("latent_split: scratch too small")
    _run("latent_split", load_library("latent").kp_latent_split, _ptr(qa), _ptr(cache), ctypes.c_longlong(cache.shape[0]), _ptr(block_table),
         block_table.shape[1], _ptr(row_seg), _ptr(positions), _ptr(scratch), int(max_context), _ptr(u), ctypes.c_float(scale), page_size, n, H,
         rankp, W, dtype_code(qa.dtype), int(USE_TC_LATENT), STREAM)
    LAUNCHES[0] += 1
    return u


def latent_prefill_ok(q: torch.Tensor, key_cols: int, value_cols: int) -> bool:
    return q.dtype == torch.bfloat16 and key_cols <= LATENT_PREFILL_MAX[0] and value_cols <= LATENT_PREFILL_MAX[1]


def latent_gather(cache: torch.Tensor, block_table: torch.Tensor, ctx_base: torch.Tensor, n_rows: int, page_size: int) -> torch.Tensor:
    """The cache rows of whole contexts side by side: row ``ctx_base[i] + t`` is key t of segment i."""
    _need(cache, "cache", torch.bfloat16); _need(block_table, "block_table", torch.int32); _need(ctx_base, "ctx_base", torch.int32)
    W = cache.shape[-1]
    n_seg = block_table.shape[0]
    if tuple(cache.shape[1:]) != (1, 1, page_size, W) or ctx_base.numel() != n_seg + 1:
        raise KernelError("latent_gather: shape mismatch")
    out = torch.empty((n_rows, W), dtype=cache.dtype, device=cache.device)
    _run("latent_gather", load_library("latent").kp_latent_gather, _ptr(cache), _ptr(block_table), block_table.shape[1], _ptr(ctx_base), n_seg,
         _ptr(out), n_rows, page_size, W, STREAM)
    return out


def latent_prefill_tc_ok(q: torch.Tensor, ex: torch.Tensor, dimp: int, rotp: int, vdimp: int) -> bool:
    """Can the tcgen05 form of the expanded pass take this call?"""
    return (USE_TC_LATENT and q.dtype == torch.bfloat16 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0 and ex.stride(0) % 8 == 0
            and bool(load_library("latent").kp_latent_prefill_tc_ok(dimp, rotp, vdimp)))


def latent_prefill_tc(q: torch.Tensor, ex: torch.Tensor, rows: torch.Tensor, rankp: int, dimp: int, rotp: int, vdimp: int,
                      cu_rows: torch.Tensor, seg_pos: torch.Tensor, big_tile_seg: torch.Tensor, big_tile_row0: torch.Tensor,
                      ctx_base: torch.Tensor, out: torch.Tensor, scale: float, H: int, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """As :func:`latent_prefill`, over tiles of 128 rows, on the tcgen05 tensor cores; ``gate`` [n, H vdimp] (rows may be strided):
    the output leaves times ``sigmoid(gate)``."""
    _need(q, "q", torch.bfloat16, contiguous=False); _need(ex, "ex", torch.bfloat16); _need(rows, "rows", torch.bfloat16)
    _need(out, "out", torch.bfloat16, contiguous=False)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (big_tile_seg, "tile_seg"), (big_tile_row0, "tile_row0"), (ctx_base, "ctx_base")):
        _need(t, nm, torch.int32)
    n = q.shape[0]
    if (q.shape[1] != H * (dimp + rotp) or tuple(out.shape) != (n, H * vdimp) or ex.shape[1] != H * (dimp + vdimp)
            or rows.shape[0] != ex.shape[0] or rows.shape[1] < rankp + rotp or big_tile_seg.numel() != big_tile_row0.numel()):
        raise KernelError("latent_prefill_tc: shape mismatch")
    if gate is not None:
        _need(gate, "gate", torch.bfloat16, contiguous=False)
        if gate.shape != out.shape:
            raise KernelError("latent_prefill_tc: gate shape")
    _run("latent_prefill_tc", load_library("latent").kp_latent_prefill_tc, _ptr(q), _rows_2d(q, "q"), n, _ptr(ex), ex.shape[1], H * dimp, _ptr(rows),
         rows.shape[0], rows.shape[1], rankp, dimp, rotp, vdimp, _ptr(cu_rows), _ptr(seg_pos), _ptr(big_tile_seg), _ptr(big_tile_row0), _ptr(ctx_base),
         big_tile_seg.numel(), _ptr(gate), _rows_2d(gate, "gate") if gate is not None else 0, _ptr(out), _rows_2d(out, "out"), ctypes.c_float(scale), H,
         STREAM)
    return out


def latent_prefill(q: torch.Tensor, ex: torch.Tensor, rows: torch.Tensor, rankp: int, dimp: int, rotp: int, vdimp: int,
                   cu_rows: torch.Tensor, seg_pos: torch.Tensor, tile_seg: torch.Tensor, tile_row0: torch.Tensor, ctx_base: torch.Tensor,
                   out: torch.Tensor, scale: float, H: int) -> torch.Tensor:
    """Causal attention of prompt portions over expanded latents: ``q`` [n, H (dimp + rotp)] (rows may be strided), ``ex`` [T, H
    dimp + H vdimp] the expanded keys and values and ``rows`` [T, W] the gathered cache rows (the rotp columns behind the first
    rankp are the shared key part), T the contexts of ``ctx_base``; tiles of 64 rows as attention_prefill takes them."""
    _need(q, "q", torch.bfloat16, contiguous=False); _need(ex, "ex", torch.bfloat16); _need(rows, "rows", torch.bfloat16)
    _need(out, "out", torch.bfloat16, contiguous=False)
    for t, nm in ((cu_rows, "cu_rows"), (seg_pos, "seg_pos"), (tile_seg, "tile_seg"), (tile_row0, "tile_row0"), (ctx_base, "ctx_base")):
        _need(t, nm, torch.int32)
    n = q.shape[0]
    if (q.shape[1] != H * (dimp + rotp) or tuple(out.shape) != (n, H * vdimp) or ex.shape[1] != H * (dimp + vdimp)
            or rows.shape[0] != ex.shape[0] or rows.shape[1] < rankp + rotp or tile_seg.numel() != tile_row0.numel()):
        raise KernelError("latent_prefill: shape mismatch")
    _run("latent_prefill", load_library("latent").kp_latent_prefill, _ptr(q), _rows_2d(q, "q"), _ptr(ex), ex.shape[1], H * dimp, _ptr(rows),
         rows.shape[1], rankp, dimp, rotp, vdimp, _ptr(cu_rows), _ptr(seg_pos), _ptr(tile_seg), _ptr(tile_row0), _ptr(ctx_base), tile_seg.numel(), _ptr(out),
         _rows_2d(out, "out"), ctypes.c_float(scale), H, STREAM)
    return out


# ---------------------------------------------------------------- skinny gemm

SKINNY_MAX_M = 64
EPI_SWIGLU = 3
EPI_ACT = 6


def skinny_ok(a: torch.Tensor, w: torch.Tensor) -> bool:
    """Can the weight-streaming kernel take this product?"""
    return (a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and a.shape[0] <= SKINNY_MAX_M
            and a.shape[1] % 32 == 0 and a.stride(1) == 1 and w.stride(1) == 1 and a.stride(0) % 8 == 0
            and w.stride(0) % 8 == 0 and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


USE_TC = True              # bfloat16 products of more than 64 rows (and some of fewer) run on tcgen05 tensor cores


TC_HEAD_FROM_M = 2         # rows from which a 65536-row head goes to the tcgen05 kernel (measured: one row ties)
TC_SPLIT_FROM_M = 17       # rows from which every product goes to the tcgen05 kernel (cut along K where that pays)


def tc_pays_for_few_rows(M: int, N: int, swiglu: bool) -> bool:
    """Few-row products that the tcgen05 kernel runs faster than the weight-streaming
    kernels (measured on B200, K = 2048, inside a decode step): the 65536-row head from
    2 rows on (a step of 2 rows 638 -> 602 us, of 4 rows 661 -> 624; one row ties), every
    product from 17 rows on (there the kernel cuts the product along K: a step of 64 rows
    1600 -> 1320 us), and below that wide products from 32 rows on."""
    if M >= TC_SPLIT_FROM_M:
        return True
    if swiglu:
        return N >= 8192 and M >= 32        # gate/up 11264 x 2048: 19.9 us against 22.9 at 32 rows, 19.8 against 32.1 at 64
    return (N >= 32768 and M >= TC_HEAD_FROM_M) or (N >= 4096 and M >= 32)


def tc_ok(a: torch.Tensor, w: torch.Tensor) -> bool:
    """Can the tcgen05 kernel take this product (bfloat16, 16-byte aligned rows, K a multiple of 8)?"""
    return (USE_TC and a.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and a.shape[1] % 8 == 0
            and a.stride(1) == 1 and w.stride(1) == 1 and a.stride(0) % 8 == 0 and w.stride(0) % 8 == 0
            and a.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


def gemm_tc(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: Optional[torch.Tensor] = None,
            accumulate: bool = False, swiglu: bool = False, split: bool = True, activation: str = "silu",
            glu: Optional[Tuple[float, float, float]] = None, plain_activation: Optional[str] = None) -> torch.Tensor:
    """out = a @ w.T (+ bias) on the tcgen05 tensor cores (TMA-fed, accumulator in tensor memory); with
    ``swiglu`` ``w`` holds gate rows then up rows and out = silu(gate) * up (or ``activation``; with ``glu`` =
    (limit, alpha, shift) the gated unit with limits of :func:`glu_clamped`).  With ``split`` a product of 17 to
    1024 rows is cut along K where that brings fewer bytes into the busiest SM (the parts of a tile are a
    thread-block cluster and are added in a fixed order)."""
    _need(a, "a", torch.bfloat16, contiguous=False); _need(w, "w", torch.bfloat16, contiguous=False)
    _need(out, "out", contiguous=False)
    M, K = a.shape
    N = w.shape[0]
    n_out = N // 2 if swiglu else N
    if w.shape[1] != K or out.shape != (M, n_out):
        raise KernelError(f"gemm_tc: shapes a{tuple(a.shape)} w{tuple(w.shape)} out{tuple(out.shape)}")
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() != N:
            raise KernelError("gemm_tc: bias size")
    lib = load_library("gemm_tc")
    if swiglu and glu is not None:
        epi = _skinny_epilogue(out, accumulate, swiglu) | (ACT_GLU_CLAMPED << 8)
        _run("gemm_tc", lib.kp_gemm_tc_split_glu, _ptr(a), _rows_2d(a, "a"), _ptr(w), _rows_2d(w, "w"), _ptr(bias), _ptr(out),
             _rows_2d(out, "out"), M, N, K, epi, 1 if split else 0, *_glu_floats(glu), STREAM, tag=f" {N}x{K}",
             work=_gemm_work(M, N, K, a, w, out))
        return out
    epi = _skinny_epilogue(out, accumulate, swiglu) | (_fused_activation(activation) << 8 if swiglu else 0)
    if plain_activation is not None:
        epi = _plain_epilogue(epi, plain_activation)
    _run("gemm_tc", lib.kp_gemm_tc_split, _ptr(a), _rows_2d(a, "a"), _ptr(w), _rows_2d(w, "w"), _ptr(bias), _ptr(out),
         _rows_2d(out, "out"), M, N, K, epi, 1 if split else 0, STREAM, tag=f" {N}x{K}",
         work=_gemm_work(M, N, K, a, w, out))
    return out


STREAM_MAX_M = 64          # rows up to which the bulk-copy kernel is preferred
USE_STREAM = True         # few-row products go to the bulk-copy kernel where their shape fits it


def stream_fits(K: int, swiglu: bool) -> bool:
    """The bulk-copy kernel streams W in chunks of 512 columns."""
    return K >= 512 and K % 512 == 0


def stream_pays(N: int, K: int) -> bool:
    """Measured on B200 (8 rows, back to back in a graph): the bulk-copy kernel wins or ties with the
    register-streaming kernel for the layer products (6144 x 2048: 8.0 against 8.1 us; gate/up 11264 x 2048:
    9.5 against 16.0; 2048 x 5632: 10.2 against 8.9; 2048 x 2048: 4.6 against 4.4) and, because its producer
    fills the ring before it waits for the kernel before it, overlaps that kernel's tail inside a model step.
    It loses on the huge grid of a 65536-row head (65 against 48 us)."""
    return N <= 16384


CONV_STEP_MAX_M = 16       # rows up to which the conv step runs in in_proj's epilogue (measured: batch 8 703 -> 672 us a
                           # step, batch 16 776 -> 741; at 64 rows the tensor-core in_proj and the separate conv kernel win)


def conv_step_fusable(a: torch.Tensor, w_in: torch.Tensor, conv_k: int) -> bool:
    """Can the weight-streaming kernel run the conv step of a decode step in in_proj's epilogue?"""
    return (USE_STREAM and skinny_ok(a, w_in) and a.shape[0] <= CONV_STEP_MAX_M and stream_fits(a.shape[1], False)
            and w_in.shape[0] % 3 == 0 and 2 <= conv_k <= 16)


def gemm_stream_conv_step(a: torch.Tensor, w_in: torch.Tensor, bias: Optional[torch.Tensor], conv_w: torch.Tensor,
                          conv_bias: Optional[torch.Tensor], state: torch.Tensor, seg_pos: torch.Tensor,
                          seg_slot: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``out = C * conv(B * X)`` for one-row segments, with ``[B | C | X] = a @ w_in.T (+ bias)`` never written
    out: the product's tile holds the matching rows of B, C and X and its epilogue runs the conv step and the
    state update of :func:`shortconv_decode` (same arithmetic, same bits)."""
    _need(a, "a", torch.bfloat16, contiguous=False); _need(w_in, "w_in", torch.bfloat16, contiguous=False)
    _need(out, "out", torch.bfloat16, contiguous=False)
    _need(conv_w, "conv_w", torch.float32); _need(state, "state", torch.float32)
    _need(seg_pos, "seg_pos", torch.int32); _need(seg_slot, "seg_slot", torch.int32)
    M, K = a.shape
    N = w_in.shape[0]
    d, conv_k = N // 3, conv_w.shape[1]
    if (w_in.shape[1] != K or N != 3 * d or out.shape != (M, d) or conv_w.shape[0] != d
            or tuple(state.shape[1:]) != (conv_k - 1, d) or seg_pos.numel() != M or seg_slot.numel() != M):
        raise KernelError("gemm_stream_conv_step: shape mismatch")
    for t, nm, n in ((bias, "bias", N), (conv_bias, "conv_bias", d)):
        if t is not None:
            _need(t, nm, torch.float32)
            if t.numel() != n:
                raise KernelError(f"gemm_stream_conv_step: {nm} size")
    lib = load_library("gemm_stream")
    _run("gemm_stream_conv_step", lib.kp_gemm_stream_conv_step, _ptr(a), _rows_2d(a, "a"), _ptr(w_in), _rows_2d(w_in, "w_in"),
         _ptr(bias), _ptr(out), _rows_2d(out, "out"), M, N, K, _ptr(conv_w), _ptr(conv_bias), _ptr(state), _ptr(seg_pos),
         _ptr(seg_slot), conv_k, STREAM, tag=f" {N}x{K}", work=_gemm_work(M, N, K, a, w_in, out))
    return out


FUSED_ACTIVATIONS = ("silu", "relu", "gelu_tanh")     # what the products' gated epilogues compute themselves
ACT_GLU_CLAMPED = 3        # the epilogues' code of the gated unit with limits (csrc/common.cuh); its constants travel beside it


def _glu_floats(glu):
    limit, alpha, shift = glu
    if not limit > 0:
        raise KernelError("the gated unit's limit must be positive")
    return ctypes.c_float(limit), ctypes.c_float(alpha), ctypes.c_float(shift)


def _fused_activation(name: str) -> int:
    if name not in FUSED_ACTIVATIONS:
        raise KernelError(f"the gated epilogue computes {', '.join(FUSED_ACTIVATIONS)}, not '{name}'")
    return activation_code(name)


def _plain_epilogue(epi: int, activation: str) -> int:
    if epi != EPI_STORE:
        raise KernelError("an ungated activation goes with a product stored in bfloat16")
    return EPI_ACT | (plain_activation_code(activation) << 8)


def _skinny_epilogue(out: torch.Tensor, accumulate: bool, swiglu: bool) -> int:
    if swiglu:
        if out.dtype != torch.bfloat16:
            raise KernelError("gemm_skinny: the SwiGLU epilogue writes bfloat16")
        return EPI_SWIGLU
    if accumulate:
        if out.dtype != torch.float32:
            raise KernelError("gemm_skinny: accumulation needs a float32 output")
        return EPI_ACCUM_F32
    if out.dtype == torch.bfloat16:
        return EPI_STORE
    if out.dtype == torch.float32:
        return EPI_STORE_F32
    raise KernelError("gemm_skinny: output dtype")


def gemm_skinny(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, bias: Optional[torch.Tensor] = None,
                accumulate: bool = False, swiglu: bool = False, activation: str = "silu",
                glu: Optional[Tuple[float, float, float]] = None, plain_activation: Optional[str] = None) -> torch.Tensor:
    """out = a @ w.T (+ bias) for up to 64 rows of bfloat16 ``a``.  With
    ``swiglu`` ``w`` holds gate rows then up rows and out = silu(gate) * up (or ``activation``; with ``glu`` =
    (limit, alpha, shift) the gated unit with limits of :func:`glu_clamped`)."""
    _need(a, "a", torch.bfloat16, contiguous=False); _need(w, "w", torch.bfloat16, contiguous=False)
    _need(out, "out", contiguous=False)
    M, K = a.shape
    N = w.shape[0]
    n_out = N // 2 if swiglu else N
    if w.shape[1] != K or out.shape != (M, n_out):
        raise KernelError(f"gemm_skinny: shapes a{tuple(a.shape)} w{tuple(w.shape)} out{tuple(out.shape)}")
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() != N:
            raise KernelError("gemm_skinny: bias size")
    if swiglu:
        if out.dtype != torch.bfloat16:
            raise KernelError("gemm_skinny: the SwiGLU epilogue writes bfloat16")
        epi = EPI_SWIGLU | ((ACT_GLU_CLAMPED if glu is not None else _fused_activation(activation)) << 8)
    elif accumulate:
        if out.dtype != torch.float32:
            raise KernelError("gemm_skinny: accumulation needs a float32 output")
        epi = EPI_ACCUM_F32
    elif out.dtype == torch.bfloat16:
        epi = EPI_STORE
    elif out.dtype == torch.float32:
        epi = EPI_STORE_F32
    else:
        raise KernelError("gemm_skinny: output dtype")
    if plain_activation is not None:
        epi = _plain_epilogue(epi, plain_activation)
    consts = _glu_floats(glu) if swiglu and glu is not None else ()
    if USE_STREAM and stream_fits(K, swiglu) and stream_pays(N, K) and M <= STREAM_MAX_M:
        lib = load_library("gemm_stream")
        _run("gemm_stream", lib.kp_gemm_stream_glu if consts else lib.kp_gemm_stream, _ptr(a), _rows_2d(a, "a"), _ptr(w),
             _rows_2d(w, "w"), _ptr(bias), _ptr(out), _rows_2d(out, "out"), M, N, K, epi, *consts, STREAM, tag=f" {N}x{K}",
             work=_gemm_work(M, N, K, a, w, out))
        return out
    lib = load_library("gemm_skinny")
    _run("gemm_skinny", lib.kp_gemm_skinny_glu if consts else lib.kp_gemm_skinny, _ptr(a), _rows_2d(a, "a"), _ptr(w),
         _rows_2d(w, "w"), _ptr(bias), _ptr(out), _rows_2d(out, "out"), M, N, K, epi, *consts, STREAM, tag=f" {N}x{K}",
         work=_gemm_work(M, N, K, a, w, out))
    return out


# ------------------------------------------------------------------ mixture of experts

MOE_MAX_TOP = 32           # experts a row can use
MOE_MAX_GROUPS = 64        # groups of experts a choice can be made from
MOE_MAX_EXPERTS = 1536     # experts the routing kernels hold in shared memory


def moe_layout_ints(n: int, E: int, top: int) -> int:
    """int32 words of the device-side layout of one step (see :func:`moe_route`)."""
    return 3 * (E + 1) + 2 * n * top


MOE_ROUTINGS = {"top_logits": 0, "softmax_all": 1, "sigmoid": 2}


def _moe_routing(routing: str) -> int:
    try:
        return MOE_ROUTINGS[routing]
    except KeyError:
        raise KernelError(f"moe: routing '{routing}' (expected one of {', '.join(MOE_ROUTINGS)})") from None


def _moe_groups(groups):
    return (0, 0) if groups is None else (int(groups[0]), int(groups[1]))


def moe_route(logits: torch.Tensor, top: int, idx: torch.Tensor, weights: torch.Tensor, layout: torch.Tensor,
              bias: Optional[torch.Tensor] = None, routing: str = "top_logits", scale: float = 1.0,
              n_identity: int = 0, groups: Optional[Tuple[int, int]] = None, renormalise: bool = False) -> None:
    """Router logits [n, E] (float32) -> the ``top`` experts of every row (``idx`` int32 [n, top], largest
    first, the lower index on ties), their weights (float32 [n, top]) and the
    layout of the (row, choice) pairs by expert (``layout``, int32, :func:`moe_layout_ints` words), which the
    grouped products read.  Nothing returns to the host.  ``routing`` ``top_logits``: the largest logits (+ ``bias``),
    weighted by the softmax over the chosen logits alone; ``softmax_all``: scores = softmax over all E outputs, the
    largest score + ``bias`` are chosen and weighted by their score times ``scale``; ``sigmoid``: the largest logits
    are chosen and each weighted by its own ``sigmoid(logit)`` times ``scale``.  The last ``n_identity``
    outputs stand for experts without weights (places in the layout, no tiles).  With ``softmax_all``: ``groups`` =
    (count, keep) lets only experts of the ``keep`` best of ``count`` equal groups of neighbours be chosen (a group is as
    good as its best expert), ``renormalise`` divides the chosen scores by their sum before ``scale``."""
    _need(logits, "logits", torch.float32); _need(idx, "idx", torch.int32); _need(weights, "weights", torch.float32)
    _need(layout, "layout", torch.int32)
    n, E = logits.shape
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() != E:
            raise KernelError("moe_route: bias size")
    if not (1 <= top <= min(E, MOE_MAX_TOP)) or E > MOE_MAX_EXPERTS:
        raise KernelError(f"moe_route: top={top} of {E} experts is not supported (top <= {MOE_MAX_TOP}, experts <= {MOE_MAX_EXPERTS})")
    if idx.numel() != n * top or weights.numel() != n * top or layout.numel() < moe_layout_ints(n, E, top):
        raise KernelError("moe_route: output sizes")
    _run("moe_route", load_library("moe").kp_moe_route, _ptr(logits), _ptr(bias), n, E, top, _moe_routing(routing),
         ctypes.c_float(scale), int(n_identity), *_moe_groups(groups), int(bool(renormalise)), _ptr(idx), _ptr(weights), _ptr(layout),
         STREAM)
    LAUNCHES[0] += 1


MOE_TC_MIN_PAIRS = [512]   # (row, expert) pairs of a step from which the experts' products run on tcgen05 tiles


def moe_set_tc_min_pairs(v: int) -> None:
    """For measurements and tests: the number of pairs from which the tcgen05 path is taken."""
    MOE_TC_MIN_PAIRS[0] = int(v)
    load_library("moe").kp_moe_set_tc_min_pairs(ctypes.c_longlong(int(v)))


def moe_tc_status() -> int:
    return _read_one("moe", "moe_tc")


def moe_router_ok(d: int, E: int) -> bool:
    """Can the fused router kernel take rows of ``d`` elements and ``E`` experts (a row, its logits and its scores in shared memory)?"""
    return d % 4 == 0 and E <= MOE_MAX_EXPERTS and (d + 2 * E) * 4 <= 200 * 1024


def moe_router(h: torch.Tensor, w_router: torch.Tensor, bias: Optional[torch.Tensor], top: int, idx: torch.Tensor,
               weights: torch.Tensor, layout: torch.Tensor, routing: str = "top_logits", scale: float = 1.0,
               n_identity: int = 0, groups: Optional[Tuple[int, int]] = None, renormalise: bool = False) -> None:
    """The router in one go: logits ``h w_router^T`` in float32 (``w_router`` [E, d] and ``bias`` are float32;
    ``h`` is widened from its storage type), the choice and the layout as :func:`moe_route` leaves them."""
    _need(h, "h", contiguous=False); _need(w_router, "w_router", torch.float32)
    _need(idx, "idx", torch.int32); _need(weights, "weights", torch.float32); _need(layout, "layout", torch.int32)
    n, d = h.shape
    E = w_router.shape[0]
    if bias is not None:
        _need(bias, "bias", torch.float32)
        if bias.numel() != E:
            raise KernelError("moe_router: bias size")
    if w_router.shape[1] != d or not moe_router_ok(d, E) or not (1 <= top <= min(E, MOE_MAX_TOP)):
        raise KernelError("moe_router: sizes not supported")
    if idx.numel() != n * top or weights.numel() != n * top or layout.numel() < moe_layout_ints(n, E, top):
        raise KernelError("moe_router: output sizes")
    _run("moe_router", load_library("moe").kp_moe_router, _ptr(h), _rows_2d(h, "h"), _ptr(w_router), _ptr(bias), n, E, d, top,
         _moe_routing(routing), ctypes.c_float(scale), int(n_identity), *_moe_groups(groups), int(bool(renormalise)), _ptr(idx), _ptr(weights), _ptr(layout),
         dtype_code(h.dtype), STREAM,
         work=(2 * n * E * d, n * d * h.element_size() + E * d * 4))
    LAUNCHES[0] += 1


def moe_experts(h: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor, layout: torch.Tensor,
                weights: torch.Tensor, top: int, out: torch.Tensor, activation: str = "silu", n_identity: int = 0,
                idx: Optional[torch.Tensor] = None, weight_input: bool = False) -> torch.Tensor:
    """out[r] += sum_j weights[r, j] * Wd_e (act(Wg_e h[r]) * (Wu_e h[r])), e = the j-th expert of row r as laid out
    by :func:`moe_route`.  ``w_gate_up``: [E, 2 ff, d] (gate rows, then up rows); ``w_down``: [E, d, ff]; ``out``
    float32 [n, d].  bfloat16 operands run on the tensor cores, float32 ones on the CUDA cores in true 32-bit.
    With ``n_identity`` the router had that many outputs more than there are experts here; a pair that chose one of
    them (``idx`` [n, top] says so) adds ``weight * h[r]``.  ``weight_input``: the weight multiplies the unit's
    input instead, ``out[r] += sum_j Wd_e (act(Wg_e w_j h[r]) * (Wu_e w_j h[r]))`` (the product ``w_j h[r]`` in
    float32, rounded to the storage type as a matrix operand)."""
    _need(h, "h", contiguous=False); _need(w_gate_up, "w_gate_up", h.dtype); _need(w_down, "w_down", h.dtype)
    _need(layout, "layout", torch.int32); _need(weights, "weights", torch.float32); _need(out, "out", torch.float32)
    n, d = h.shape
    E_real, ff2, d2 = w_gate_up.shape
    E = E_real + int(n_identity)
    ff = ff2 // 2
    if d2 != d or ff2 != 2 * ff or tuple(w_down.shape) != (E_real, d, ff) or tuple(out.shape) != (n, d):
        raise KernelError("moe_experts: shape mismatch")
    if weights.numel() != n * top or layout.numel() < moe_layout_ints(n, E, top):
        raise KernelError("moe_experts: routing tables do not fit")
    if n_identity:
        _need(idx, "idx", torch.int32)
        if idx.numel() != n * top:
            raise KernelError("moe_experts: idx size")
        if weight_input:
            raise KernelError("moe_experts: weights on the inputs do not go with identity experts")
    act = torch.empty((n * top, ff), dtype=h.dtype, device=h.device)
    y = torch.empty((n * top, d), dtype=torch.float32, device=h.device)
    # (many rows, 16-bit: the tcgen05 tiles read the rows laid out place by place)
    hs = (torch.empty((n * top, d), dtype=h.dtype, device=h.device)
          if (weight_input or (h.dtype == torch.bfloat16 and n * top >= MOE_TC_MIN_PAIRS[0])) else None)
    _run("moe_experts", load_library("moe").kp_moe_experts_weighted, _ptr(h), _rows_2d(h, "h"), _ptr(w_gate_up), _ptr(w_down), _ptr(layout),
         _ptr(weights), _ptr(act), _ptr(y), _ptr(out), _ptr(hs), n, E, top, d, ff, activation_code(activation), dtype_code(h.dtype),
         int(n_identity), _ptr(idx if n_identity else None), int(bool(weight_input)), STREAM, tag=f" {E}x{ff}x{d}",
         work=(6 * n * top * ff * d, min(E, n * top) * 3 * ff * d * h.element_size()))     # (bytes: the experts a step can touch)
    LAUNCHES[0] += 2
    return out
