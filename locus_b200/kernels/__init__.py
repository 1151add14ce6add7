"""Python entry points of the hand-written CUDA kernels.

Each function takes torch tensors that already live on the GPU, checks what the C entry
point cannot check (devices, contiguity, element types, shapes), and launches on torch's
current stream through ctypes.  Nothing here allocates device memory or falls back to
another implementation: a missing or failing kernel module raises.

The functions are the only way the parts reach the GPU, so a test may replace them by
plain torch functions of the same signature to exercise the engine's host logic.
"""
from __future__ import annotations

import ctypes
from typing import Optional, Tuple

import torch

from ..csrc import build as _build

ERR_UNSUPPORTED = 10001

_DT = {torch.float32: 0, torch.bfloat16: 1}


class KernelError(RuntimeError):
    pass


def dtype_code(dt: torch.dtype) -> int:
    try:
        return _DT[dt]
    except KeyError:
        raise KernelError(f"element type {dt} is not supported by the kernels (float32, bfloat16)") from None


_LIBS = {}


def _lib(name: str) -> ctypes.CDLL:
    lib = _LIBS.get(name)
    if lib is None:
        lib = _LIBS[name] = _build.load(name)
    return lib


def _p(t: Optional[torch.Tensor]):
    return None if t is None else ctypes.c_void_p(t.data_ptr())


_stream_override = None


def _stream():
    if _stream_override is not None:
        return _stream_override
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


class pdl_scope:
    """Within the scope, kernels that support it are launched with programmatic dependent
    launch (see csrc/common.cuh): the next kernel's blocks are scheduled while the previous
    kernel still runs.  Used for the CUDA graphs of decode steps."""

    def __enter__(self):
        for lib in _LIBS.values():
            if hasattr(lib, "locus_set_pdl"):
                lib.locus_set_pdl(1)
        return self

    def __exit__(self, *exc):
        for lib in _LIBS.values():
            if hasattr(lib, "locus_set_pdl"):
                lib.locus_set_pdl(0)
        return False


class stream_scope:
    """Within the scope every launch goes to the stream that is torch's current stream when
    the scope is entered (looked up once instead of once per launch)."""

    def __enter__(self):
        global _stream_override
        self._saved = _stream_override
        _stream_override = ctypes.c_void_p(torch.cuda.current_stream().cuda_stream) if torch.cuda.is_available() else None
        return self

    def __exit__(self, *exc):
        global _stream_override
        _stream_override = self._saved
        return False


class kernel_times:
    """Opt-in table of where the time of eager steps goes, by entry point of this module (the reference has no
    profiler of its own: it prints counters at exit and is timed from outside).  Inside the scope an event is
    recorded behind every entry point's launch, on the stream it went to, and the launch is charged the time from
    the event before it on that stream (the scope's start, for the first launch on the stream that opened the
    scope) to its own: its run and whatever the stream waited for in front of it.  ``ModelRunner.step`` replays no
    graph meanwhile.  ``table()`` waits for the device and returns {entry point: (launches, milliseconds)}; the
    first launch on another stream is counted without a time."""

    def __enter__(self):
        global _TIMES
        _need(_TIMES is None, "kernel_times: scopes do not nest")
        self._spans = []   # (entry point, event before, event behind)
        self._counts = {}
        self._last = {}    # stream -> the event behind its latest launch
        start = torch.cuda.Event(enable_timing=True)
        start.record()
        self._last[torch.cuda.current_stream().cuda_stream] = start
        _TIMES = self
        return self

    def __exit__(self, *exc):
        global _TIMES
        _TIMES = None
        return False

    def _mark(self, what: str) -> None:
        ev = torch.cuda.Event(enable_timing=True)
        ev.record()
        key = torch.cuda.current_stream().cuda_stream
        before = self._last.get(key)
        if before is not None:
            self._spans.append((what, before, ev))
        self._counts[what] = self._counts.get(what, 0) + 1
        self._last[key] = ev

    def restart(self) -> None:
        """The current stream starts a stretch of work of its own (a side stream that has just been told to wait
        for the main one): its next launch is charged from here, not from its last launch long ago."""
        ev = torch.cuda.Event(enable_timing=True)
        ev.record()
        self._last[torch.cuda.current_stream().cuda_stream] = ev

    def table(self) -> dict:
        torch.cuda.synchronize()
        ms = {}
        for what, a, b in self._spans:
            ms[what] = ms.get(what, 0.0) + a.elapsed_time(b)
        return {what: (n, ms.get(what, 0.0)) for what, n in self._counts.items()}


_TIMES: Optional[kernel_times] = None


def timing_active() -> bool:
    """Whether a :class:`kernel_times` scope is open (steps then run eagerly)."""
    return _TIMES is not None


def timing_restart() -> None:
    """See :meth:`kernel_times.restart`; nothing without an open scope."""
    if _TIMES is not None:
        _TIMES.restart()


# kernels launched through this module since import (some entry points launch two and count the second themselves)
launches = 0
_LAUNCHES_OF = {}
MOE_SORT_ONE_LAUNCH_EXPERTS = 40 * 1024 // (9 * 4)   # up to this many experts moe_sort is one launch, else two


def _count_launches(n: int) -> None:
    global launches
    launches += n


def _check(code: int, what: str, detail: str = "") -> None:
    global launches
    if code == 0:
        launches += _LAUNCHES_OF.get(what, 1)
        if _TIMES is not None:
            _TIMES._mark(what)
        return
    if code == ERR_UNSUPPORTED:
        raise KernelError(f"{what}: sizes or element types outside what the kernel takes {detail}")
    raise KernelError(f"{what}: CUDA error {code} {detail}")


def _need(cond: bool, msg: str) -> None:
    if not cond:
        raise KernelError(msg)


def _cuda_c(t: torch.Tensor, name: str) -> None:
    _need(t.is_cuda, f"{name} must be a CUDA tensor")
    _need(t.is_contiguous(), f"{name} must be contiguous")


def _i32(t: torch.Tensor, name: str) -> None:
    _cuda_c(t, name)
    _need(t.dtype == torch.int32, f"{name} must be int32")


LL = ctypes.c_longlong
I = ctypes.c_int
F = ctypes.c_float


# ---------------------------------------------------------------------------
def embed_rows(tokens: torch.Tensor, table: torch.Tensor, out: torch.Tensor, copies: int = 1, scale: float = 1.0,
               dyt_norm=None, positions: Optional[torch.Tensor] = None, pos_table: Optional[torch.Tensor] = None,
               keep: Optional[torch.Tensor] = None) -> None:
    """out[t, :] = table[tokens[t], :] * scale as float32; ``copies`` > 1: the row that many times, one behind the
    other (``out`` [T, copies * H]).  ``dyt_norm`` = (alpha, weight, bias): the row through :func:`dyt`'s norm.
    ``pos_table`` [positions, H] with ``positions`` [T] int32: row positions[t] is added behind the factor.  ``keep`` [T, H]
    float32: the rows once more."""
    _i32(tokens, "tokens")
    _cuda_c(table, "table")
    _cuda_c(out, "out")
    T, H = out.shape[0], table.shape[1]
    _need(out.dtype == torch.float32, "embed_rows: out must be float32")
    _need(tokens.numel() == T and copies >= 1 and out.shape[1] == H * copies, "embed_rows: shape mismatch")
    if pos_table is not None:
        _cuda_c(pos_table, "pos_table")
        _need(positions is not None and pos_table.shape[1] == H and positions.numel() >= T, "embed_rows: positions and their table")
        _i32(positions, "positions")
    if keep is not None:
        _cuda_c(keep, "keep")
        _need(keep.dtype == torch.float32 and tuple(keep.shape) == (T, H), "embed_rows: keep must be float32 [T, H]")
    code = _lib("elementwise").locus_embed_rows(
        _p(tokens), _p(table), I(dtype_code(table.dtype)), _p(out), I(T), I(H), I(copies), F(scale),
        *_dyt_args(dyt_norm, H), _p(positions), _p(pos_table), I(dtype_code(pos_table.dtype) if pos_table is not None else 0),
        _p(keep), _stream()
    )
    _check(code, "embed_rows")


def _dyt_args(norm, H: int):
    """(alpha, weight, bias, element type) of a Dynamic Tanh norm for the entry points; None: no norm."""
    if norm is None:
        return None, None, None, I(0)
    alpha, w, b = norm
    for t, n in ((alpha, 1), (w, H), (b, H)):
        _need(t.is_cuda and t.is_contiguous() and t.numel() == n and t.dtype == w.dtype,
              "dyt: alpha [1], weight and bias [H] of one element type on the device")
    return _p(alpha), _p(w), _p(b), I(dtype_code(w.dtype))


def dyt(x: torch.Tensor, norm=None, out: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None,
        add=None) -> None:
    """Dynamic Tanh, D(z) = tanh(alpha z) * weight + bias elementwise, ``norm`` = (alpha, weight, bias): out[i] = D(u) with
    u = x[rows[i] if rows else i] (float32 rows).  ``add`` = (y, (alpha, weight, bias), scale or None): u = x + scale *
    D_y(y) instead, D_y with those parameters and ``y`` rows like ``x``; without ``rows`` u is written back to ``x``.
    ``out`` may be absent (only the addition), or ``x`` itself (neither ``rows`` nor ``add``)."""
    _f32c(x, "dyt: x")
    H = x.shape[-1]
    n = x.shape[0] if out is None else out.shape[0]
    _need(x.is_contiguous() and (out is not None or add is not None) and (norm is None) == (out is None), "dyt: norm and out go together")
    if out is not None:
        _cuda_c(out, "out")
        _need(out.shape[-1] == H, "dyt: out width")
        _need(out.data_ptr() != x.data_ptr() or (rows is None and add is None), "dyt: out is x")
    if rows is not None:
        _i32(rows, "rows")
        _need(rows.numel() == n and out is not None, "dyt: rows/out mismatch")
    else:
        _need(x.shape[0] >= n, "dyt: x/out mismatch")
    y = ls = None
    y_norm = None
    if add is not None:
        y, y_norm, ls = add
        _f32c(y, "dyt: y")
        _need(y.is_contiguous() and y.shape[-1] == H and y.shape[0] >= (x.shape[0] if rows is not None else n), "dyt: y rows")
        if ls is not None:
            _cuda_c(ls, "scale")
            _need(ls.numel() == H, "dyt: scale [H]")
    code = _lib("elementwise").locus_dyt(
        _p(x), _p(y), *_dyt_args(y_norm, H), _p(ls), I(dtype_code(ls.dtype) if ls is not None else 0), _p(out),
        I(dtype_code(out.dtype) if out is not None else 0), *_dyt_args(norm, H), _p(rows), I(n), I(H), _stream())
    _check(code, "dyt")


def rmsnorm_adds(x: torch.Tensor) -> bool:
    """Whether :func:`rmsnorm` can fold a pending addition into rows like ``x``'s."""
    return x.dtype == torch.float32 and x.shape[-1] % 4 == 0


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, out: torch.Tensor,
            rows: Optional[torch.Tensor] = None, add=None, add_rows: Optional[torch.Tensor] = None) -> None:
    """out[i] = x[rows[i] if rows else i] * rsqrt(mean(x^2) + eps) * w  (statistics in float32).

    ``add`` = (pair_out, pair_pos, top_k): first x[i] += the sum that :func:`moe_combine` forms (same
    order), written back to ``x``; needs :func:`rmsnorm_adds`.  With ``rows`` the sum enters the norm
    of the gathered rows only and ``x`` stays as it was.  ``add_rows`` (float32 rows like ``x``'s): added in the same way,
    behind that sum."""
    _cuda_c(x, "x")
    _cuda_c(w, "w")
    _cuda_c(out, "out")
    H = x.shape[-1]
    n = out.shape[0]
    _need(w.numel() == H and out.shape[-1] == H, "rmsnorm: width mismatch")
    if rows is not None:
        _i32(rows, "rows")
        _need(rows.numel() == n, "rmsnorm: rows/out mismatch")
    else:
        _need(x.shape[0] == n, "rmsnorm: x/out mismatch")
    add_src = add_pos = None
    add_k = 0
    if add is not None:
        add_src, add_pos, add_k = add
        _need(rmsnorm_adds(x), "rmsnorm: cannot fold the expert sum into these rows")
        _cuda_c(add_src, "pair_out")
        _i32(add_pos, "pair_pos")
        _need(add_src.dtype in (torch.float32, torch.bfloat16) and add_src.shape[-1] == H
              and add_pos.numel() >= (n if rows is None else x.shape[0]) * add_k,
              "rmsnorm: expert sum of another shape")
    if add_rows is not None:
        _cuda_c(add_rows, "add_rows")
        _need(rmsnorm_adds(x) and add_rows.dtype == torch.float32 and add_rows.shape == x.shape, "rmsnorm: add_rows must be float32 rows like x's")
    code = _lib("elementwise").locus_rmsnorm(
        _p(x), I(dtype_code(x.dtype)), _p(w), I(dtype_code(w.dtype)), F(eps), _p(out),
        I(dtype_code(out.dtype)), _p(rows), I(n), I(H), _p(add_src),
        I(dtype_code(add_src.dtype) if add_src is not None else 0), _p(add_pos), I(add_k), _p(add_rows), _stream()
    )
    _check(code, "rmsnorm")


class ExpertLayout:
    """Device tensors that lay (token, slot) pairs out by expert (see :func:`moe_sort`)."""

    MIN_TILE = 8

    def __init__(self, n_pairs_max: int, n_experts: int, tile_m: int, device) -> None:
        """``tile_m``: rows of a tile; :func:`moe_sort` may be given another one per call
        (at least ``MIN_TILE``), the buffers are sized for the smallest."""
        self.tile_m = tile_m
        self.n_experts = n_experts
        self.max_tiles = (n_pairs_max + self.MIN_TILE - 1) // self.MIN_TILE + n_experts
        i32 = dict(dtype=torch.int32, device=device)
        self.counts = torch.zeros(n_experts, **i32)
        self.offsets = torch.zeros(n_experts + 1, **i32)
        self.sorted_pair = torch.zeros(n_pairs_max, **i32)
        self.pair_pos = torch.zeros(n_pairs_max, **i32)
        self.tile_expert = torch.zeros(self.max_tiles, **i32)
        self.tile_row0 = torch.zeros(self.max_tiles, **i32)
        self.tile_rows = torch.zeros(self.max_tiles, **i32)
        self.n_tiles = torch.zeros(1, **i32)
        # a second tile list over the same rows, with tiles of tile2_m rows (0: none; see moe_sort)
        self.tile2_m = 0
        self.tile2_expert = torch.zeros(self.max_tiles, **i32)
        self.tile2_row0 = torch.zeros(self.max_tiles, **i32)
        self.tile2_rows = torch.zeros(self.max_tiles, **i32)
        self.n_tiles2 = torch.zeros(1, **i32)

    def tiles_for(self, n_pairs: int, tile_m: Optional[int] = None) -> int:
        """Upper bound of the number of row tiles (of ``tile_m`` rows, default the layout's) when ``n_pairs``
        pairs are routed."""
        return min(self.max_tiles, n_pairs // (tile_m or self.tile_m) + min(n_pairs, self.n_experts) + 1)


# Tests switch this off to run the CUDA-core product on bfloat16 inputs.
USE_TENSOR_CORES = True


def tensor_cores_take(x: torch.Tensor, w: torch.Tensor, x_rows: Optional[torch.Tensor] = None) -> bool:
    """Whether :func:`linear` runs this product on the tensor cores: bfloat16 activations and
    weights, rows that TMA can address (width and row stride multiples of 8 elements,
    16-byte aligned base), and no row gather (gather into a buffer first)."""
    K = x.shape[-1]
    return (USE_TENSOR_CORES and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and x_rows is None
            and K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


FEW_ROWS = 8  # rows of x per tile of the row-streaming kernel


def few_rows_take(x: torch.Tensor, w: torch.Tensor, m: int, layout: Optional["ExpertLayout"] = None) -> bool:
    """Whether :func:`linear` runs this product with the row-streaming kernel: at most 8 rows
    (per expert tile when grouped), width a multiple of 8, 32-byte aligned rows."""
    K = x.shape[-1]
    rows_ok = layout.tile_m <= FEW_ROWS if layout is not None else m <= FEW_ROWS
    return (rows_ok and K % 8 == 0 and x.stride(0) % 8 == 0 and x.data_ptr() % 32 == 0 and w.data_ptr() % 32 == 0)


# Most rows of a plain product that go to the weight-streaming tensor-core kernel (it takes up to 32, and
# expert tiles of 8, 16 or 32 rows).  The four dense products of a layer at the A2.7B sizes take 46 us with
# either kernel at 16 rows; at 24 rows 59 us there and 47 us on the tcgen05 kernel (cut along K where it has
# few tiles), at 32 rows 61 and 47.
SKINNY_ROWS = 16
SKINNY_TILE_ROWS = 32  # largest expert tile of that kernel's grouped form
SKINNY_MIN_ROWS = 1


def skinny_takes(x: torch.Tensor, w: torch.Tensor, m: int, layout: Optional["ExpertLayout"] = None) -> bool:
    """Whether :func:`linear` runs this product with the weight-streaming tensor-core kernel:
    bfloat16 x bfloat16, at most ``SKINNY_ROWS`` rows (per expert tile of 8, 16 or 32 rows when grouped)."""
    K = x.shape[-1]
    if layout is not None:
        rows_ok = layout.tile_m in (8, 16, 32)
    else:
        rows_ok = SKINNY_MIN_ROWS <= m <= SKINNY_ROWS
    return (USE_TENSOR_CORES and rows_ok and x.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and K % 8 == 0
            and x.stride(0) % 8 == 0 and x.data_ptr() % 16 == 0 and w.data_ptr() % 16 == 0)


_N_SM = 0


def _sm_count() -> int:
    global _N_SM
    if _N_SM == 0:
        _N_SM = torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
    return _N_SM


SPLIT_SCRATCH_BYTES = 64 << 20   # float32 partial sums of a product split along K
_PLANS: dict = {}
_SPLIT_SCRATCH: dict = {}


def token_tile(m: int, dual: bool = False, n_weight_tiles: int = 0, k: int = 0) -> int:
    """Token tile of a plain product on the tensor cores (see :func:`tc_plan`)."""
    return tc_plan(m, n_weight_tiles * 128, k, dual)[0]


def tc_plan(m: int, n: int, k: int, dual: bool) -> Tuple[int, int]:
    """(token tile, splits along K) of a plain product of ``m`` rows with an [n, k] weight on the
    tcgen05 kernel.  While a tile waits for its weights its time hardly depends on its tokens (measured at
    k = 2048, one tile per SM: 12.7 us with 32 tokens, 13.5 with 64, 15 with 128, 18.3 with 256: 0.38 us
    + 0.75 ns per token for every 64 of k), so what counts is how many rounds the tiles make over the SMs,
    and a product with few tiles (a 2048-row weight has 16) leaves most SMs idle unless it is also cut
    along k; the partial sums then cost a second kernel.  The plan with the least estimated time wins."""
    key = (m, n, k, dual)
    plan = _PLANS.get(key)
    if plan is not None:
        return plan
    top = 128 if dual else 256
    cands = [t for t in (16, 32, 64, 128, 256) if t <= top]
    n_w = max(1, -(-n // 128))
    if k <= 0:  # sizes unknown: the smallest tile that holds the rows
        plan = (next((t for t in cands if m <= t), top), 1)
        _PLANS[key] = plan
        return plan
    n_sm = _sm_count()
    nkb = -(-k // 64)
    best, best_cost = (top, 1), None
    for t in cands:
        if t < 32 and m > t:
            continue
        tiles = -(-m // t) * n_w
        per_kb = (0.38 + 0.00075 * t) * (1.15 if dual else 1.0)
        options = [1]
        if not dual and n % 4 == 0 and tiles * 2 <= n_sm and nkb >= 8:
            s_max = min(n_sm // tiles, nkb // 2, 16, SPLIT_SCRATCH_BYTES // (4 * m * n))
            options += [s for s in range(2, s_max + 1)]
        for sp in options:
            kb = -(-nkb // sp)
            sp = -(-nkb // kb)
            rounds = -(-(tiles * sp) // n_sm)
            cost = rounds * (0.5 + kb * per_kb)
            if sp > 1:
                # the second kernel and its reading of the partial sums (fitted: 64 x 2048 x 2048 in 8 parts
                # takes 9.4 us, 256 x 6144 x 2048 in 3 parts 17.4 us)
                cost += 6.5 + sp * m * n * 4 / 3.5e6
            if best_cost is None or cost < best_cost - 1e-9 or (abs(cost - best_cost) <= 1e-9 and t > best[0]):
                best, best_cost = (t, sp), cost
        if m <= t:
            break
    _PLANS[key] = best
    return best


def _split_scratch(device) -> torch.Tensor:
    """The partial sums' buffer of the stream that launches: products on different streams (the shared expert
    beside the routed ones) must not share one.  Made at a stream's first split product, which is never inside
    a graph capture: a step is run once in the open before it is captured."""
    key = (device, _stream().value)
    t = _SPLIT_SCRATCH.get(key)
    if t is None:
        t = torch.empty(SPLIT_SCRATCH_BYTES // 4, dtype=torch.float32, device=device)
        _SPLIT_SCRATCH[key] = t
    return t


def expert_second_tile(n_pairs: int, n_experts: int) -> int:
    """Row tile of the experts' SECOND product (one accumulator per tile: 256 token rows fit the tensor memory)
    when it pays to walk the layout in larger tiles than the first product's 128, else 0.  With 137 rows per expert
    on average half of the experts need a second 128-row tile, which costs nearly what a full one costs (the tile
    waits for the same weights): measured at 60 x (2048 -> 2048), 4 picks, 2,048 tokens 122 us with 128-row tiles and
    110 us with 256-row tiles, at 64 x (3584 -> 2560), 8 picks 396 and 351 us; at 512 tokens (34 rows per expert)
    87 and 95 us."""
    return 256 if n_pairs >= 96 * n_experts else 0


def expert_tile(n_pairs: int, n_experts: int) -> int:
    """Row tile of a grouped product on the tensor cores.  Always the full 128 rows: a tile reads its
    tokens through a box that fits the rows it really has (16 to 256), so a tile with few rows costs little,
    and every expert's weights stream once.  Measured on the routed experts of 60 x (2048 -> 1408 -> 2048),
    4 picks: 75 us for 8 tokens, 148 us for 32, 173 us for 64, 181 us for 512, 238 us for 2,048 (the
    weight-streaming kernel with tiles of 8 to 32 rows: 79, 167, 219, 626 us)."""
    return 128


# activations of a product's epilogue, by their code in the kernels' flags
ACTIVATIONS = {None: 0, "relu2": 1, "glu_clamp": 2, "softcap": 3, "reglu": 4}


def tc_error() -> int:
    """Error word of the tensor-core module (0 = fine); reading it synchronises the device.
    Non-zero: a bounded wait inside a kernel ran out (1 producer, 2 MMA, 3 epilogue)."""
    return int(_lib("gemm_tc").locus_gemm_tc_error())


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor, *, w2: Optional[torch.Tensor] = None,
           bias: Optional[torch.Tensor] = None, accumulate: bool = False,
           row_scale: Optional[torch.Tensor] = None, scale_rows: Optional[torch.Tensor] = None,
           x_rows: Optional[torch.Tensor] = None, x_row_div: int = 1, layout: Optional[ExpertLayout] = None,
           n_rows: Optional[int] = None, lists_ready: bool = False, second_tiles: bool = False,
           act: Optional[str] = None, act_limit: float = 0.0, act_scale: float = 1.0) -> None:
    """out = x . w^T with float32 accumulation on CUDA cores (see csrc/gemm_simt.cu).

    ``w2``: out = silu(x . w^T) * (x . w2^T).  ``act`` = "relu2": out = max(x . w^T + bias, 0)^2 (not with ``w2``).
    ``act`` = "glu_clamp" (with ``w2``): the clamped gated unit out = g sigmoid(1.702 g) (u + 1) with g = min(s x . w^T,
    ``act_limit``), u = clamp(s x . w2^T, -act_limit, act_limit), where s is the row's ``row_scale`` (1 without): the
    scale then stands for a factor on the row of x and is not applied once more behind the activation.  ``act`` =
    "reglu" (with ``w2``): max(x . w^T + b, 0) * (x . w2^T + b2), ``bias`` being [2 N], b and behind it b2.  ``act`` =
    "softcap" (not with ``w2``): ``act_limit`` * tanh(``act_scale`` * v / ``act_limit``) behind everything else.  ``bias`` [N] is added, ``row_scale`` [M]
    multiplies the row (``scale_rows``: row m uses row_scale[scale_rows[m]]), ``accumulate`` adds the result into the float32 ``out``.
    ``x_rows``: logical row m reads x[x_rows[m] // x_row_div].  ``layout``: grouped product,
    ``w`` is [E, N, K] and logical rows are the expert-sorted pairs of the layout.
    ``n_rows``: number of logical rows (default: rows of ``out``).  ``lists_ready``: the layout was filled by a
    kernel that finished before the kernel in front of this one started (the experts' second product), so a
    kernel launched with programmatic dependent launch may read it before it waits for the one in front.
    ``second_tiles``: a grouped product on the tensor cores walks the layout's second tile list (``moe_sort`` with
    ``tile2_m``) instead of the first.
    """
    # (x may be a stretch of columns of wider rows: the kernels take its row stride)
    _need(x.is_cuda and x.stride(-1) == 1 and (x.is_contiguous() or x.dim() == 2), "linear: x must be CUDA rows with unit stride")
    _cuda_c(w, "w")
    _cuda_c(out, "out")
    K = x.shape[-1]
    N = w.shape[-2]
    _need(w.shape[-1] == K, f"linear: x has width {K} but w has {w.shape[-1]}")
    _need(out.shape[-1] == N, f"linear: out has width {out.shape[-1]} but w has {N} rows")
    M = out.shape[0] if n_rows is None else n_rows
    _need(M <= out.shape[0], "linear: more rows than out holds")
    if x_rows is None and layout is None:
        _need(x.shape[0] >= M, "linear: x has fewer rows than out")
    if w2 is not None:
        _need(w2.shape == w.shape and w2.dtype == w.dtype and w2.is_contiguous(), "linear: w2 must match w")
    if accumulate:
        _need(out.dtype == torch.float32, "linear: accumulate needs a float32 out")
    _need(act in ACTIVATIONS and not (act == "relu2" and w2 is not None) and not (act == "reglu" and w2 is None) and not (act == "glu_clamp" and (w2 is None or not act_limit > 0))
          and not (act == "softcap" and (w2 is not None or not act_limit > 0)),
          f"linear: activation {act!r} (known: relu2 without w2; reglu with w2; glu_clamp with w2 and a positive act_limit; softcap without "
          "w2 and with a positive act_limit)")
    flags = I((1 if accumulate else 0) | (ACTIVATIONS[act] << 1))
    if bias is not None:
        _need(bias.numel() == (2 * N if act == "reglu" else N) and bias.is_contiguous(), "linear: bias size")
    if row_scale is not None:
        _need(row_scale.dtype == torch.float32 and row_scale.is_contiguous(), "linear: row_scale must be float32")
        if scale_rows is not None:
            _i32(scale_rows, "scale_rows")
        else:
            _need(row_scale.numel() >= M, "linear: row_scale must hold M rows")
    if x_rows is not None:
        _i32(x_rows, "x_rows")
    if layout is not None:
        # a layout may count experts without weights behind the ones with (their tiles are taken off its lists:
        # moe_identity)
        _need(w.dim() == 3 and w.shape[0] <= layout.n_experts, "linear: grouped product needs w [E, N, K]")
    if skinny_takes(x, w, M, layout):
        # bfloat16, up to 32 rows per tile: weight-streaming tensor-core kernel (csrc/gemm_skinny.cu)
        if layout is not None:
            tile = layout.tile_m
            te, t0, tr, nt = layout.tile_expert, layout.tile_row0, layout.tile_rows, layout.n_tiles
            max_tiles, stride = layout.tiles_for(M), N * K
        else:
            _need(w.dim() == 2, "linear: w must be [N, K]")
            tile = 8 if M <= 8 else (16 if M <= 16 else 32)
            te = t0 = tr = nt = None
            max_tiles = stride = 0
        code = _lib("gemm_skinny").locus_gemm_skinny(
            _p(x), _p(w), _p(w2), _p(bias), I(dtype_code(bias.dtype) if bias is not None else 0), _p(out),
            I(dtype_code(out.dtype)), flags, F(act_limit), F(act_scale), _p(row_scale), _p(scale_rows), _p(x_rows),
            I(x_row_div), I(M), I(N), I(K), LL(x.stride(0)), LL(out.stride(0)), I(tile), _p(te), _p(t0), _p(tr),
            _p(nt), I(max_tiles), LL(stride), I(1 if (lists_ready and layout is not None) else 0), _stream()
        )
        _check(code, "linear", f"(skinny; M={M}, N={N}, K={K}, tile {tile})")
        return
    if few_rows_take(x, w, M, layout):
        # a handful of rows: bandwidth-bound row-streaming kernel (csrc/gemv.cu)
        if layout is not None:
            te, t0, tr, nt = layout.tile_expert, layout.tile_row0, layout.tile_rows, layout.n_tiles
            max_tiles, stride = layout.tiles_for(M), N * K
        else:
            _need(w.dim() == 2, "linear: w must be [N, K]")
            te = t0 = tr = nt = None
            max_tiles = stride = 0
        code = _lib("gemv").locus_gemv(
            _p(x), I(dtype_code(x.dtype)), _p(w), _p(w2), I(dtype_code(w.dtype)), _p(bias),
            I(dtype_code(bias.dtype) if bias is not None else 0), _p(out), I(dtype_code(out.dtype)),
            flags, F(act_limit), F(act_scale), _p(row_scale), _p(scale_rows), _p(x_rows), I(x_row_div), I(M), I(N), I(K),
            LL(x.stride(0)), LL(out.stride(0)), _p(te), _p(t0), _p(tr), _p(nt), I(max_tiles), LL(stride), _stream()
        )
        _check(code, "linear", f"(few rows; M={M}, N={N}, K={K}, x {x.dtype}, w {w.dtype})")
        return
    if tensor_cores_take(x, w, x_rows):
        # bfloat16 x bfloat16: tcgen05 kernel (csrc/gemm_tc.cu)
        if layout is not None and second_tiles and layout.tile2_m > 0:
            TN, splits, scratch = layout.tile2_m, 1, None
            te, t0, tr, nt = layout.tile2_expert, layout.tile2_row0, layout.tile2_rows, layout.n_tiles2
            max_tiles = layout.tiles_for(M, layout.tile2_m)
        elif layout is not None:
            TN, splits, scratch = layout.tile_m, 1, None
            te, t0, tr, nt = layout.tile_expert, layout.tile_row0, layout.tile_rows, layout.n_tiles
            max_tiles = layout.tiles_for(M)
        else:
            _need(w.dim() == 2, "linear: w must be [N, K]")
            TN, splits = tc_plan(M, N, K, w2 is not None)
            if act and splits > 1:
                # the activation belongs behind the whole sum: such a product is not cut along K
                TN, splits = tc_plan(M, N, K, True)[0], 1
            if splits > 1:
                scratch = _split_scratch(x.device)
            te = t0 = tr = nt = None
            max_tiles = 0
        code = _lib("gemm_tc").locus_gemm_tc(
            _p(x), LL(M), LL(x.stride(0)), _p(w), _p(w2), LL(w.numel() // K), _p(bias),
            I(dtype_code(bias.dtype) if bias is not None else 0), _p(out), I(dtype_code(out.dtype)),
            flags, F(act_limit), F(act_scale), _p(row_scale), _p(scale_rows), I(M), I(N), I(K), LL(out.stride(0)), I(TN),
            _p(te), _p(t0), _p(tr), _p(nt), I(max_tiles), _p(scratch if splits > 1 else None), I(splits), _stream()
        )
        if splits > 1 and code == 0:
            _count_launches(1)   # the kernel that adds the splits up
        _check(code, "linear", f"(tensor cores; M={M}, N={N}, K={K}, token tile {TN}, {splits} splits)")
        return
    if layout is not None:
        _need(layout.tile_m == 64, "linear: the CUDA-core product uses 64-row tiles")
        te, t0, tr, nt = layout.tile_expert, layout.tile_row0, layout.tile_rows, layout.n_tiles
        max_tiles = layout.tiles_for(M)
        stride = N * K
    else:
        _need(w.dim() == 2, "linear: w must be [N, K]")
        te = t0 = tr = nt = None
        max_tiles = 0
        stride = 0
    code = _lib("gemm_simt").locus_gemm_simt(
        _p(x), I(dtype_code(x.dtype)), _p(w), _p(w2), I(dtype_code(w.dtype)), _p(bias),
        I(dtype_code(bias.dtype) if bias is not None else 0), _p(out), I(dtype_code(out.dtype)),
        flags, F(act_limit), F(act_scale), _p(row_scale), _p(scale_rows), _p(x_rows), I(x_row_div), I(M), I(N), I(K),
        LL(x.stride(0)), LL(out.stride(0)), _p(te), _p(t0), _p(tr), _p(nt), I(max_tiles), LL(stride),
        _stream()
    )
    _check(code, "linear", f"(M={M}, N={N}, K={K}, x {x.dtype}, w {w.dtype})")


def rope_kv_write(qkv: torch.Tensor, positions: torch.Tensor, inv_freq: Optional[torch.Tensor],
                  q_out: torch.Tensor, pool: torch.Tensor, slots: torch.Tensor, *, n_heads: int,
                  n_kv_heads: int, head_dim: int, rot_dim: int, interleaved: bool,
                  page_tokens: int, write_kv: bool = True) -> None:
    """Rotate q and k by position, write q to ``q_out`` and k, v into the layer's pages.

    ``pool`` is one layer's pages [n_pages, 2, n_kv_heads, page_tokens, head_dim];
    ``slots[t] = page * page_tokens + offset``.  ``inv_freq`` None: no rotation.
    """
    _cuda_c(qkv, "qkv")
    _cuda_c(q_out, "q_out")
    _cuda_c(pool, "pool")
    _i32(positions, "positions")
    _i32(slots, "slots")
    T = qkv.shape[0]
    _need(qkv.shape[1] == (n_heads + 2 * n_kv_heads) * head_dim, "rope_kv_write: qkv width")
    _need(qkv.dtype == q_out.dtype == pool.dtype, "rope_kv_write: q, k, v and the cache share one element type")
    _need(tuple(pool.shape[1:]) == (2, n_kv_heads, page_tokens, head_dim), "rope_kv_write: pool layout")
    _need(positions.numel() >= T and slots.numel() >= T and q_out.shape[0] >= T, "rope_kv_write: T mismatch")
    if inv_freq is not None:
        _need(inv_freq.dtype == torch.float32 and inv_freq.numel() == rot_dim // 2 and inv_freq.is_cuda,
              "rope_kv_write: inv_freq must be float32 [rot_dim / 2]")
    code = _lib("elementwise").locus_rope_kv_write(
        _p(qkv), I(dtype_code(qkv.dtype)), _p(positions), _p(inv_freq), _p(q_out), _p(pool),
        _p(slots), I(T), I(n_heads), I(n_kv_heads), I(head_dim), I(rot_dim),
        I(1 if interleaved else 0), I(page_tokens), I(1 if write_kv else 0), _stream()
    )
    _check(code, "rope_kv_write")


def _sink_args(sink, n_heads: int):
    """(flag, pointer) of a softmax sink for the attention entry points: ``sink`` is False (none), True (one more term of
    score 0) or a float32 tensor [n_heads] of learned scores."""
    if isinstance(sink, torch.Tensor):
        _need(sink.is_cuda and sink.dtype == torch.float32 and sink.is_contiguous() and sink.numel() == n_heads,
              "attention: a learned sink must be float32 [n_heads] on the device")
        return I(1), _p(sink)
    return I(1 if sink else 0), None


def _slopes_arg(slopes: Optional[torch.Tensor], n_heads: int):
    """Pointer of a distance bias's slopes (float32 [n_heads] on the device; None: no bias)."""
    if slopes is not None:
        _need(slopes.is_cuda and slopes.dtype == torch.float32 and slopes.is_contiguous() and slopes.numel() == n_heads,
              "attention: the slopes of a distance bias must be float32 [n_heads] on the device")
    return _p(slopes)


def attn_chunk(q: torch.Tensor, pool: torch.Tensor, out: torch.Tensor, *, seg_q0: torch.Tensor,
               seg_qn: torch.Tensor, seg_ctx: torch.Tensor, block_table: torch.Tensor,
               items: torch.Tensor, n_items: int, n_heads: int, n_kv_heads: int, head_dim: int,
               page_tokens: int, window: int, scale: float, keep_first: int = 0, sink=False, chunk: int = 0,
               slopes: Optional[torch.Tensor] = None) -> None:
    """Attention of portions of prompts: ``items`` [n_items, 2] = (segment, first query of a
    16-query tile).  Keys come from the cache through ``block_table`` [n_seg, width].  ``keep_first``: with a
    window, a request's first that many tokens stay in sight of every later query; ``sink``: the softmax has one
    more term in its denominator that has no value: True for the score 0, a float32 tensor [n_heads] for a learned
    score per head (taken as it is, not multiplied by ``scale``).  ``chunk`` > 0 (without a window): a query sees the keys of
    its own chunk of that many positions, counted from position 0, up to itself.  ``slopes`` [n_heads] float32: a distance
    bias, slopes[h] * (p - t) is taken off the scaled score of a query at position p with the key at t."""
    _cuda_c(q, "q")
    _cuda_c(out, "out")
    _cuda_c(pool, "pool")
    _i32(block_table, "block_table")
    _i32(items, "items")
    _need(q.dtype == pool.dtype == out.dtype, "attn_chunk: q, cache and out share one element type")
    code = _lib("attention").locus_attn_chunk(
        _p(q), I(dtype_code(q.dtype)), _p(pool), _p(out), _p(seg_q0), _p(seg_qn), _p(seg_ctx),
        _p(block_table), I(block_table.shape[1]), _p(items), I(n_items), I(n_heads), I(n_kv_heads),
        I(head_dim), I(page_tokens), I(window), I(chunk), F(scale), I(keep_first), *_sink_args(sink, n_heads),
        _slopes_arg(slopes, n_heads), _stream()
    )
    _check(code, "attn_chunk", f"(heads {n_heads}/{n_kv_heads}, head_dim {head_dim})")


MMA_HEAD_DIMS = tuple(range(16, 257, 16))
MMA_QUERY_TILE = 64


def attn_chunk_mma_takes(q: torch.Tensor, head_dim: int) -> bool:
    """Whether the tensor-core kernel of prompt portions takes this case (bfloat16, head size
    in ``MMA_HEAD_DIMS``); otherwise :func:`attn_chunk` does it on the CUDA cores."""
    return USE_TENSOR_CORES and q.dtype == torch.bfloat16 and head_dim in MMA_HEAD_DIMS


MMA_ATTN_MAX_SPLITS = 16


def attn_chunk_mma_scratch(head_dim: int) -> Tuple[int, int]:
    """Floats of the two scratch buffers (sums; maxima and denominators) that :func:`attn_chunk_mma` needs
    to cut the keys of a step with few 64-query tiles into ranges (at most two blocks per SM are made)."""
    units = 2 * _sm_count() + MMA_ATTN_MAX_SPLITS
    return units * MMA_QUERY_TILE * head_dim, units * MMA_QUERY_TILE * 2


def attn_chunk_mma_splits(n_items: int, n_heads: int, max_ctx: int) -> int:
    """Ranges the keys of every item are cut into: enough for two blocks per SM when the step has fewer
    blocks than SMs (a short portion behind a long context), down to one tile of 64 keys per range.  A block
    takes about 1.9 us per key tile and the merge 2.5 us, so from four tiles on the cut pays: 64 tokens behind
    1,024 take 35 us in one range and 11 us in 16; 52 behind 30,000, 880 us and 91 us."""
    blocks = n_items * n_heads
    n_sm = _sm_count()
    tiles = -(-max_ctx // MMA_QUERY_TILE)
    if blocks >= n_sm or tiles < 4:
        return 1
    return max(1, min(MMA_ATTN_MAX_SPLITS, (2 * n_sm) // blocks, tiles))


def attn_chunk_mma(q: torch.Tensor, pool: torch.Tensor, out: torch.Tensor, *, seg_q0: torch.Tensor,
                   seg_qn: torch.Tensor, seg_ctx: torch.Tensor, block_table: torch.Tensor,
                   items: torch.Tensor, n_items: int, n_heads: int, n_kv_heads: int, head_dim: int,
                   page_tokens: int, window: int, scale: float, n_splits: int = 1,
                   part_o: Optional[torch.Tensor] = None, part_ml: Optional[torch.Tensor] = None,
                   keep_first: int = 0, sink=False, chunk: int = 0, slopes: Optional[torch.Tensor] = None) -> None:
    """Attention of portions of prompts on the tensor cores: ``items`` [n_items, 2] =
    (segment, first query of a 64-query tile); otherwise as :func:`attn_chunk`.  ``n_splits`` > 1
    (:func:`attn_chunk_mma_splits`) with scratch of :func:`attn_chunk_mma_scratch` floats: the keys of
    every item are cut into that many ranges, merged in ascending order by a second kernel."""
    _cuda_c(q, "q")
    _cuda_c(out, "out")
    _cuda_c(pool, "pool")
    _i32(block_table, "block_table")
    _i32(items, "items")
    _need(q.dtype == pool.dtype == out.dtype == torch.bfloat16, "attn_chunk_mma: bfloat16 only")
    if n_splits > 1:
        units = n_items * n_heads * n_splits
        _need(part_o is not None and part_ml is not None and part_o.dtype == part_ml.dtype == torch.float32
              and part_o.numel() >= units * MMA_QUERY_TILE * head_dim and part_ml.numel() >= units * MMA_QUERY_TILE * 2,
              "attn_chunk_mma: scratch too small for these ranges")
    code = _lib("attention_mma").locus_attn_chunk_mma(
        _p(q), _p(pool), _p(out), _p(seg_q0), _p(seg_qn), _p(seg_ctx), _p(block_table), I(block_table.shape[1]),
        _p(items), I(n_items), I(n_heads), I(n_kv_heads), I(head_dim), I(page_tokens), I(window), I(chunk), F(scale),
        I(n_splits), _p(part_o if n_splits > 1 else None), _p(part_ml if n_splits > 1 else None), I(keep_first),
        *_sink_args(sink, n_heads), _slopes_arg(slopes, n_heads), _stream()
    )
    if n_splits > 1 and code == 0:
        _count_launches(1)
    _check(code, "attn_chunk_mma", f"(heads {n_heads}/{n_kv_heads}, head_dim {head_dim}, {n_splits} key ranges)")


TC_ATTN_HEAD_DIM = 128   # the tcgen05 attention kernel: this head size, pages of a multiple of 64 tokens
TC_ATTN_MIN_TOKENS = 256  # from this many new tokens in a step on, the tcgen05 kernel takes every portion


def attn_chunk_tc_takes(q: torch.Tensor, head_dim: int, page_tokens: int, n_tokens: int, max_ctx: int = 0) -> bool:
    """Whether the tcgen05 kernel of prompt portions takes this step: bfloat16, head size 128, pages of a
    multiple of 64 tokens, and either enough new tokens to fill blocks of 128 queries or a context long enough
    that the kernel's faster walk over the keys (cut into ranges, :func:`attn_chunk_tc_splits`) outweighs its
    start-up.  Measured at 16 heads against the mma.sync kernel, both with their key ranges: 128 new tokens
    behind 1,000 / 4,000 / 30,000 cached ones 18.6 / 20.4 / 59.6 us against 15.0 / 31.5 / 153.8 us; 16 new tokens
    14.2 / 16.4 / 53.9 us against 9.0 / 17.4 / 89.4 us."""
    if not (USE_TENSOR_CORES and q.dtype == torch.bfloat16 and head_dim == TC_ATTN_HEAD_DIM and page_tokens % 64 == 0):
        return False
    return n_tokens >= TC_ATTN_MIN_TOKENS or max_ctx >= (2048 if n_tokens >= 128 else 4096)


TC_ATTN_MAX_SPLITS = 16
TC_ATTN_QUERY_BLOCK = 128   # queries of a block of the tcgen05 kernel (two of the 64-query tiles of its item list)


def attn_chunk_tc_splits(n_items: int, n_heads: int, max_ctx: int, n_rows: int = 0) -> int:
    """Ranges the key tiles of every block of :func:`attn_chunk_tc` are cut into.  A block takes 128 queries of one
    head, a block per SM: a portion of a few hundred tokens behind a long context makes fewer blocks than the GPU
    has SMs, each walking thousands of keys alone.  Then the keys are cut so that about every SM has a block, down
    to four tiles of 128 keys per range (a block's start and end cost about four tiles' time).  ``n_rows``: the step's tokens,
    those of other kernels' segments among them: a range keeps a partial result for each, and they must fit
    :func:`attn_chunk_tc_scratch`."""
    blocks = -(-n_items // 2) * n_heads
    n_sm = _sm_count()
    tiles = -(-max_ctx // TC_ATTN_QUERY_BLOCK)
    if 2 * blocks > n_sm or tiles < 8:
        return 1
    fit = TC_ATTN_QUERY_BLOCK * n_sm // max(1, n_rows * n_heads) if n_rows > 0 else TC_ATTN_MAX_SPLITS
    return max(1, min(TC_ATTN_MAX_SPLITS, n_sm // blocks, tiles // 4, fit))


def attn_chunk_tc_scratch() -> Tuple[int, int]:
    """Floats of the two scratch buffers (sums; maxima and denominators) that :func:`attn_chunk_tc` needs for any
    cut that :func:`attn_chunk_tc_splits` chooses: one partial result per (token, head, range), and the ranges
    never outnumber SMs / blocks while a block holds at most 128 tokens of a head."""
    units = TC_ATTN_QUERY_BLOCK * _sm_count()
    return units * TC_ATTN_HEAD_DIM, units * 2


def attn_chunk_tc(q: torch.Tensor, pool: torch.Tensor, out: torch.Tensor, *, seg_q0: torch.Tensor,
                  seg_qn: torch.Tensor, seg_ctx: torch.Tensor, block_table: torch.Tensor,
                  items: torch.Tensor, n_items: int, n_heads: int, n_kv_heads: int, head_dim: int,
                  page_tokens: int, window: int, scale: float, n_splits: int = 1,
                  part_o: Optional[torch.Tensor] = None, part_ml: Optional[torch.Tensor] = None,
                  keep_first: int = 0, sink=False, chunk: int = 0, slopes: Optional[torch.Tensor] = None) -> None:
    """Attention of portions of prompts with tcgen05 tensor cores (scores and sums in tensor memory):
    ``items`` as for :func:`attn_chunk_mma` (tiles of 64 queries; a block takes an even one and the 64 queries
    behind it).  ``n_splits`` > 1 (:func:`attn_chunk_tc_splits`) with scratch of :func:`attn_chunk_tc_scratch`
    floats: the key tiles of every block are cut into that many ranges, merged in ascending order by a second
    kernel.  ``keep_first`` (with a window): a request's first tokens stay in sight; ``sink``: one more term of score 0
    in the softmax's denominator; ``chunk``, ``slopes`` as for :func:`attn_chunk`."""
    _cuda_c(q, "q")
    _cuda_c(out, "out")
    _cuda_c(pool, "pool")
    _i32(block_table, "block_table")
    _i32(items, "items")
    _need(q.dtype == pool.dtype == out.dtype == torch.bfloat16, "attn_chunk_tc: bfloat16 only")
    _need(1 <= n_splits <= TC_ATTN_MAX_SPLITS, f"attn_chunk_tc: 1 to {TC_ATTN_MAX_SPLITS} key ranges")
    if n_splits > 1:
        units = q.shape[0] * n_heads * n_splits
        n_o, n_ml = units * TC_ATTN_HEAD_DIM, units * 2
        _need(part_o is not None and part_ml is not None and part_o.dtype == part_ml.dtype == torch.float32
              and part_o.is_cuda and part_ml.is_cuda and part_o.numel() >= n_o and part_ml.numel() >= n_ml,
              "attn_chunk_tc: scratch too small for these ranges")
    code = _lib("attention_tc").locus_attn_chunk_tc(
        _p(q), LL(q.shape[0]), _p(pool), LL(pool.shape[0]), _p(out), _p(seg_q0), _p(seg_qn), _p(seg_ctx),
        _p(block_table), I(block_table.shape[1]), _p(items), I(n_items), I(n_heads), I(n_kv_heads), I(head_dim),
        I(page_tokens), I(window), I(chunk), F(scale), I(n_splits), _p(part_o if n_splits > 1 else None),
        _p(part_ml if n_splits > 1 else None), I(keep_first if window > 0 else 0), *_sink_args(sink, n_heads),
        _slopes_arg(slopes, n_heads), _stream()
    )
    if n_splits > 1 and code == 0:
        _count_launches(1)
    _check(code, "attn_chunk_tc", f"(heads {n_heads}/{n_kv_heads}, head_dim {head_dim}, pages of {page_tokens}, "
                                  f"{n_splits} key ranges)")


def attn_chunk_tc_rows(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, out: torch.Tensor, *, seg_q0: torch.Tensor,
                       seg_qn: torch.Tensor, seg_ctx: torch.Tensor, kv_row0: torch.Tensor, items: torch.Tensor, n_items: int,
                       n_heads: int, n_kv_heads: int, head_dim: int, window: int, scale: float, n_splits: int = 1,
                       part_o: Optional[torch.Tensor] = None, part_ml: Optional[torch.Tensor] = None, keep_first: int = 0,
                       sink=False, chunk: int = 0, slopes: Optional[torch.Tensor] = None) -> None:
    """:func:`attn_chunk_tc` over keys and values in plain rows instead of pages: ``k`` and ``v`` [rows, n_kv_heads *
    head_dim] (stretches of columns of wider rows are taken), a segment's key at position t in row ``kv_row0[segment]`` + t
    of both.  ``items`` lists tiles of 64 queries of the segments that have such rows; the others' entries of ``kv_row0`` are
    not read."""
    _cuda_c(q, "q")
    _cuda_c(out, "out")
    _i32(items, "items")
    _i32(kv_row0, "kv_row0")
    _need(q.dtype == k.dtype == v.dtype == out.dtype == torch.bfloat16, "attn_chunk_tc_rows: bfloat16 only")
    for t in (k, v):
        _need(t.is_cuda and t.stride(1) == 1 and t.shape[0] == k.shape[0] and t.shape[1] == n_kv_heads * head_dim,
              "attn_chunk_tc_rows: k, v rows [rows, n_kv_heads * head_dim]")
    _need(1 <= n_splits <= TC_ATTN_MAX_SPLITS, f"attn_chunk_tc_rows: 1 to {TC_ATTN_MAX_SPLITS} key ranges")
    if n_splits > 1:
        units = q.shape[0] * n_heads * n_splits
        _need(part_o is not None and part_ml is not None and part_o.dtype == part_ml.dtype == torch.float32
              and part_o.is_cuda and part_ml.is_cuda and part_o.numel() >= units * TC_ATTN_HEAD_DIM and part_ml.numel() >= units * 2,
              "attn_chunk_tc_rows: scratch too small for these ranges")
    code = _lib("attention_tc").locus_attn_chunk_tc_rows(
        _p(q), LL(q.shape[0]), _p(k), LL(k.stride(0)), _p(v), LL(v.stride(0)), LL(k.shape[0]), _p(out), _p(seg_q0), _p(seg_qn),
        _p(seg_ctx), _p(kv_row0), _p(items), I(n_items), I(n_heads), I(n_kv_heads), I(head_dim), I(window), I(chunk), F(scale),
        I(n_splits), _p(part_o if n_splits > 1 else None), _p(part_ml if n_splits > 1 else None),
        I(keep_first if window > 0 else 0), *_sink_args(sink, n_heads), _slopes_arg(slopes, n_heads), _stream())
    if n_splits > 1 and code == 0:
        _count_launches(1)
    _check(code, "attn_chunk_tc", f"(rows; heads {n_heads}/{n_kv_heads}, head_dim {head_dim}, {n_splits} key ranges)")


def attn_tc_error() -> int:
    """Error word of the tcgen05 attention module (0 = fine); reading it synchronises the device."""
    return int(_lib("attention_tc").locus_attn_tc_error())


def attn_error() -> int:
    """Error word of the attention module (0 = fine; 1 = a decode step's ``max_splits`` did not cover its
    longest context); reading it synchronises the device and clears it."""
    return int(_lib("attention").locus_attn_error())


def attn_gqa_error() -> int:
    """Error word of the grouped-query decode attention module (0 = fine; 1 = a wait for a bulk copy ran out);
    reading it synchronises the device and clears it."""
    return int(_lib("attention_gqa").locus_attn_gqa_error())


DECODE_SPLIT = 128


USE_GQA_DECODE = True   # tests switch it off to run grouped-query models on the per-head kernels
# The range cut's cost model of the grouped-query kernel, in keys (csrc/attn_ranges.cuh): the fixed cost of a range,
# and the cost of merging one more range per query head of the group (the merging warp takes the group's heads two
# at a time).  Measured at 28 heads on 4, 8,192 keys: with 2 x 7 = 14 keys per range a call takes 50 / 51 / 52 /
# 65 / 196 us at 1 / 4 / 8 / 16 / 64 requests (2: 51 / 52 / 51 / 66 / 202; 35: 75 / 76 / 74 / 75 / 196).
GQA_COST_RANGE, GQA_COST_MERGE_PER_HEAD = 64, 2
# Fewer (request, key/value head) pairs than this: the per-head kernels, which cut the work G times finer (at 28
# heads on 4 and 8,192 keys: 25 / 37 / 55 / 96 us at 1 / 2 / 4 / 8 requests against 50 / 50 / 51 / 52).
GQA_MIN_UNITS = 16


def attn_decode_gqa_takes(dtype: torch.dtype, n_heads: int, n_kv_heads: int, head_dim: int, page_tokens: int,
                          n_items: int) -> bool:
    """Whether :func:`attn_decode` runs the grouped-query kernel (csrc/attention_gqa.cu): bfloat16, 2 to 16
    query heads per key/value head, head size 64 or 128, pages of a multiple of 16 tokens, and enough
    (request, key/value head) pairs to fill the GPU with whole groups."""
    g = n_heads // max(1, n_kv_heads)
    return (USE_GQA_DECODE and USE_TENSOR_CORES and dtype == torch.bfloat16 and n_heads % max(1, n_kv_heads) == 0
            and 2 <= g <= 16 and head_dim in (64, 128) and page_tokens % 16 == 0 and n_items <= 1024
            and n_items * n_kv_heads >= GQA_MIN_UNITS)


def decode_streams(head_dim: int, dtype: torch.dtype, page_tokens: int, max_items: int) -> bool:
    """Whether :func:`attn_decode` runs the streaming kernel (the condition of csrc/attention.cu): rows of
    64 to 512 bytes (8, 16 or 32 lanes to a row: its 16-byte pieces rounded up to a power of two), pages that
    are a multiple of that lane count's chunk of 32, 16 or 8 keys, and at most 1024 requests."""
    pieces = head_dim * (4 if dtype == torch.float32 else 2) // 16
    lanes = 0 if pieces < 4 else 8 if pieces <= 8 else 16 if pieces <= 16 else 32 if pieces <= 32 else 0
    return lanes > 0 and page_tokens % (256 // lanes) == 0 and max_items <= 1024


def decode_units(max_items: int, n_heads: int, head_dim: int, dtype: torch.dtype, max_splits: int, device,
                 page_tokens: int = 64, n_kv_heads: int = 0, fixed_ranges: bool = False) -> int:
    """How many partial results the scratch of :func:`attn_decode` should hold for batches of up to
    ``max_items`` requests.  The streaming kernels (:func:`decode_streams`, :func:`attn_decode_gqa_takes`) want
    one per (request, head) plus eight rounds of the grid's warps, so that short batches can be cut finely; the
    split kernel (other head and page sizes; and the small batches of a grouped-query model whose rows the
    per-head streaming kernel does not take) wants one per (request, head, split), ``max_splits`` being the
    splits of the longest context that the cache allows."""
    try:
        n_sm = torch.cuda.get_device_properties(device).multi_processor_count
    except Exception:  # no GPU (host tests with emulated kernels)
        n_sm = 148
    streaming = max_items * n_heads + 8 * 16 * n_sm
    if fixed_ranges:   # a window that keeps first tokens: one more range per (request, head), or the split kernel
        if decode_streams(head_dim, dtype, page_tokens, max_items):
            return streaming + max_items * n_heads
        return max(streaming + max_items * n_heads, max_items * n_heads * max_splits)
    if decode_streams(head_dim, dtype, page_tokens, max_items):
        return streaming
    if n_kv_heads > 0 and attn_decode_gqa_takes(dtype, n_heads, n_kv_heads, head_dim, page_tokens,
                                                max(max_items, GQA_MIN_UNITS)):
        # batches below GQA_MIN_UNITS pairs go to the split kernel
        small = min(max_items, max(0, -(-GQA_MIN_UNITS // n_kv_heads) - 1))
        return max(streaming, small * n_heads * max_splits)
    return max_items * n_heads * max_splits


def attn_decode_gqa_variant(few: Optional[bool]) -> None:
    """Force the grouped-query decode kernel's shape for few (request, key/value head) pairs (six warps a block,
    four chunks in flight per warp) on (True) or off (False: ten warps, two chunks), or leave the choice to the
    library (None).  For tests and measurements."""
    _lib("attention_gqa").locus_attn_decode_gqa_set_deep(I(-1 if few is None else 1 if few else 0))


def attn_decode_variant(deep: Optional[bool]) -> None:
    """Force the streaming decode kernel's variant with two chunks in flight per warp on (True) or off (False), or
    leave the choice to the library (None: by the number of (request, head) pairs and the longest context).  For
    tests and measurements."""
    _lib("attention").locus_attn_decode_set_deep(I(-1 if deep is None else 1 if deep else 0))


def attn_decode(q: torch.Tensor, pool: torch.Tensor, out: torch.Tensor, *, seg_q0: torch.Tensor,
                seg_qn: torch.Tensor, seg_ctx: torch.Tensor, block_table: torch.Tensor,
                items: torch.Tensor, n_items: int, n_heads: int, n_kv_heads: int, head_dim: int,
                page_tokens: int, window: int, scale: float, part_o: torch.Tensor,
                part_ml: torch.Tensor, counters: torch.Tensor, max_splits: int, keep_first: int = 0,
                sink=False, chunk: int = 0, slopes: Optional[torch.Tensor] = None) -> None:
    """Attention of single new tokens: ``items`` [n_items] = segments with one new token.  ``keep_first``, ``sink``, ``chunk``,
    ``slopes`` as for :func:`attn_chunk` (the streaming kernels, per head and per group of query heads, walk the kept tokens in front
    of the window as one more range of the request and want scratch for two ranges per request and head, the kernel whose
    ranges are fixed for ``max_splits``: :func:`decode_units` with ``fixed_ranges``).

    ``part_o`` (float32, units * head_dim) and ``part_ml`` (float32, 2 * units) are scratch for
    partial results, ``units`` as :func:`decode_units` gives it (at least n_items * n_heads);
    ``counters`` (int32, n_items * n_heads) must be zero before the call and is zero after it;
    ``max_splits`` must be at least longest_position // DECODE_SPLIT + 1.
    """
    _cuda_c(q, "q")
    _cuda_c(out, "out")
    _cuda_c(pool, "pool")
    _i32(block_table, "block_table")
    _i32(items, "items")
    _need(q.dtype == pool.dtype == out.dtype, "attn_decode: q, cache and out share one element type")
    _need(part_o.dtype == torch.float32 and part_ml.dtype == torch.float32, "attn_decode: float32 scratch")
    max_units = min(part_o.numel() // head_dim, part_ml.numel() // 2)
    _need(max_units >= n_items * n_heads, "attn_decode: scratch too small")
    _need(pool.numel() * pool.element_size() < (64 << 30), "attn_decode: a layer's cache pool of 64 GiB or more")
    _i32(counters, "counters")
    _need(counters.numel() >= n_items * n_heads, "attn_decode: counters too small")
    if attn_decode_gqa_takes(q.dtype, n_heads, n_kv_heads, head_dim, page_tokens, n_items):
        # several query heads per key/value head: the kernel that reads every cache row once for its whole group
        code = _lib("attention_gqa").locus_attn_decode_gqa(
            _p(q), _p(pool), _p(out), _p(seg_q0), _p(seg_ctx), _p(block_table), I(block_table.shape[1]), _p(items),
            I(n_items), I(n_heads), I(n_kv_heads), I(head_dim), I(page_tokens), I(window), I(chunk), F(scale), _p(part_o),
            _p(part_ml), _p(counters), ctypes.c_longlong(max_units), I(GQA_COST_RANGE),
            I(GQA_COST_MERGE_PER_HEAD * (n_heads // n_kv_heads)), I(keep_first if window > 0 else 0), *_sink_args(sink, n_heads),
            _slopes_arg(slopes, n_heads), _stream()
        )
        _check(code, "attn_decode", f"(grouped queries; heads {n_heads}/{n_kv_heads}, head_dim {head_dim})")
        return
    code = _lib("attention").locus_attn_decode(
        _p(q), I(dtype_code(q.dtype)), _p(pool), _p(out), _p(seg_q0), _p(seg_qn), _p(seg_ctx),
        _p(block_table), I(block_table.shape[1]), _p(items), I(n_items), I(n_heads), I(n_kv_heads),
        I(head_dim), I(page_tokens), I(window), I(chunk), F(scale), _p(part_o), _p(part_ml), _p(counters), I(max_splits),
        ctypes.c_longlong(max_units), I(keep_first if window > 0 else 0), *_sink_args(sink, n_heads), _slopes_arg(slopes, n_heads),
        _stream()
    )
    _check(code, "attn_decode", f"(heads {n_heads}/{n_kv_heads}, head_dim {head_dim})")


SCORE_FUNCTIONS = {"softmax": 0, "sigmoid": 1}
# what a group of experts is judged by when only some groups stay eligible: the sum of its two best selection scores,
# or its best one (a flag beside the score function's code, see csrc/route_select.cuh)
GROUP_SCORES = {"top2": 0, "best": 16}


def _route_rule(score_fn: str, sel_bias: Optional[torch.Tensor], n_group: int, n_group_used: int, n_experts: int,
                what: str, group_score: str = "top2"):
    """The arguments that say how experts are chosen, checked: (score code, bias pointer, groups, groups used)."""
    _need(score_fn in SCORE_FUNCTIONS, f"{what}: score function {score_fn!r} (known: {', '.join(SCORE_FUNCTIONS)})")
    _need(group_score in GROUP_SCORES, f"{what}: group score {group_score!r} (known: {', '.join(GROUP_SCORES)})")
    if sel_bias is not None:
        _need(sel_bias.is_cuda and sel_bias.dtype == torch.float32 and sel_bias.is_contiguous()
              and sel_bias.numel() == n_experts, f"{what}: the selection bias must be float32 [n_experts]")
    _need(1 <= n_group <= 32 and n_experts % n_group == 0,
          f"{what}: {n_group} groups must divide {n_experts} experts (at most 32 groups)")
    _need(n_group == 1 or 1 <= n_group_used <= n_group, f"{what}: groups used must be within 1..{n_group}")
    return I(SCORE_FUNCTIONS[score_fn] | GROUP_SCORES[group_score]), _p(sel_bias), I(n_group), I(n_group_used)


class RouterScratch:
    """Scratch of :func:`router_topk`: the router logits of a step and one counter per tile of
    8 tokens (zero between launches); ``fused_counter``: the counter of :func:`route_fused_small`."""

    def __init__(self, max_tokens: int, n_logits: int, device) -> None:
        self.max_tokens, self.n_logits = max_tokens, n_logits
        self.logits = torch.empty(max_tokens * n_logits, dtype=torch.float32, device=device)
        self.counters = torch.zeros((max_tokens + 7) // 8, dtype=torch.int32, device=device)
        self.fused_counter = torch.zeros(1, dtype=torch.int32, device=device)


def router_topk(h: torch.Tensor, w_router: torch.Tensor, w_gate: Optional[torch.Tensor],
                ids: torch.Tensor, wts: torch.Tensor, gamma: Optional[torch.Tensor], *, top_k: int,
                renorm: bool, scale: float = 1.0, scratch: Optional[RouterScratch] = None, score_fn: str = "softmax",
                sel_bias: Optional[torch.Tensor] = None, n_group: int = 1, n_group_used: int = 1,
                logit_bias: Optional[torch.Tensor] = None, group_score: str = "top2") -> None:
    """Router: scores of all experts (``score_fn``: softmax over them, or a sigmoid of each logit), top-k by
    repeated arg-max, weights; and gamma = sigmoid(w_gate . h) when the shared expert is gated.  All in float32.
    ``sel_bias`` [E] is added to the scores for the selection only; with ``n_group`` > 1 only the
    ``n_group_used`` groups of experts with the best two-score sums (``group_score`` "best": with the best single
    score) are eligible.  ``logit_bias`` [E] float32 is
    part of the logits (a router with a bias of its own): it enters the scores, the selection and the weights.
    ``scratch`` must hold T tokens of E (+1 with a gate) logits (made on the fly when None)."""
    _cuda_c(h, "h")
    _cuda_c(w_router, "w_router")
    _i32(ids, "ids")
    T, H = h.shape
    E = w_router.shape[0]
    _need(w_router.shape[1] == H, "router_topk: width mismatch")
    _need(wts.dtype == torch.float32 and wts.numel() >= T * top_k and ids.numel() >= T * top_k,
          "router_topk: ids / wts too small")
    if w_gate is not None:
        _need(w_gate.numel() == H and gamma is not None and gamma.dtype == torch.float32 and gamma.numel() >= T,
              "router_topk: gate needs w_gate [H] and gamma [T] float32")
    e1 = E + (1 if w_gate is not None else 0)
    if scratch is None:
        scratch = RouterScratch(T, e1, h.device)
    _need(scratch.n_logits >= e1 and scratch.max_tokens >= T, "router_topk: scratch too small")
    code = _lib("moe_route").locus_router_topk(
        _p(h), I(dtype_code(h.dtype)), _p(w_router), I(dtype_code(w_router.dtype)), _p(w_gate),
        I(dtype_code(w_gate.dtype) if w_gate is not None else 0), _p(scratch.logits), _p(scratch.counters),
        _p(ids), _p(wts), _p(gamma), I(T), I(H), I(E), I(top_k), I(1 if renorm else 0), F(scale),
        *_route_rule(score_fn, sel_bias, n_group, n_group_used, E, "router_topk", group_score), _p(_logit_bias(logit_bias, E)),
        _stream()
    )
    _check(code, "router_topk", f"(H={H}, E={E}, k={top_k})")


def _logit_bias(b: Optional[torch.Tensor], n: int) -> Optional[torch.Tensor]:
    if b is not None:
        _need(b.is_cuda and b.dtype == torch.float32 and b.is_contiguous() and b.numel() >= n,
              "router: the logit bias must be float32, one number per logit row")
    return b


def router_logits(h: torch.Tensor, w_all: torch.Tensor, logits: torch.Tensor,
                  bias: Optional[torch.Tensor] = None) -> None:
    """logits[t, e] = w_all[e] . h[t] (+ ``bias[e]``, float32) in float32 with the weight-streaming tensor-core kernel,
    for ANY number of tokens (tiles of up to 16): one kernel, and one order of the sum, for
    every batch shape.  bfloat16 ``h`` [T, H] and ``w_all`` [E (+1), H]; ``logits`` [T, >= E (+1)]."""
    _cuda_c(h, "h")
    _cuda_c(w_all, "w_all")
    T, H = h.shape
    n = w_all.shape[0]
    _need(h.dtype == torch.bfloat16 and w_all.dtype == torch.bfloat16 and H % 8 == 0, "router_logits: bfloat16, H % 8 == 0")
    _need(logits.dtype == torch.float32 and logits.shape[0] >= T and logits.shape[1] >= n and logits.stride(1) == 1,
          "router_logits: logits must be float32 [T, >= rows of w_all]")
    # tiles of 16 tokens from 9 tokens on: with 32 a block's chain is twice as long (64 tokens: 9.1 us against 4.2,
    # 8,192 tokens: 60 against 34), and the order of a sum does not depend on the tile
    tile = 8 if T <= 8 else 16
    code = _lib("gemm_skinny").locus_gemm_skinny(
        _p(h), _p(w_all), None, _p(_logit_bias(bias, n)), I(0), _p(logits), I(0), I(0), None, None, None, I(1), I(T), I(n), I(H),
        LL(h.stride(0)), LL(logits.stride(0)), I(tile), None, None, None, None, I(0), LL(0), I(0), _stream()
    )
    _check(code, "router_logits", f"(T={T}, H={H}, rows {n})")


def router_select(logits: torch.Tensor, n_experts: int, has_gate: bool, ids: torch.Tensor, wts: torch.Tensor,
                  gamma: Optional[torch.Tensor], *, n_tokens: int, top_k: int, renorm: bool, scale: float = 1.0,
                  score_fn: str = "softmax", sel_bias: Optional[torch.Tensor] = None, n_group: int = 1,
                  n_group_used: int = 1, group_score: str = "top2") -> None:
    """Scores from the first ``n_experts`` columns of ``logits``, top-k by repeated arg-max,
    weights (the rule of :func:`router_topk`); gamma = sigmoid(column n_experts) when ``has_gate``."""
    _need(logits.is_cuda and logits.dtype == torch.float32 and logits.stride(1) == 1, "router_select: float32 logits")
    _i32(ids, "ids")
    _need(wts.dtype == torch.float32 and wts.numel() >= n_tokens * top_k and ids.numel() >= n_tokens * top_k,
          "router_select: ids / wts too small")
    if has_gate:
        _need(gamma is not None and gamma.dtype == torch.float32 and gamma.numel() >= n_tokens, "router_select: gamma")
    code = _lib("moe_route").locus_router_select(
        _p(logits), I(logits.stride(0)), _p(ids), _p(wts), _p(gamma), I(n_tokens), I(n_experts), I(top_k),
        I(1 if has_gate else 0), I(1 if renorm else 0), F(scale),
        *_route_rule(score_fn, sel_bias, n_group, n_group_used, n_experts, "router_select", group_score), _stream()
    )
    _check(code, "router_select", f"(E={n_experts}, k={top_k})")


def moe_sort(ids: torch.Tensor, n_pairs: int, layout: ExpertLayout, tile_m: Optional[int] = None,
             tile2_m: int = 0) -> None:
    """Fill ``layout`` from the picked experts ``ids`` (first ``n_pairs`` entries), with row
    tiles of ``tile_m`` rows (default: the layout's).  ``tile2_m`` > 0: also a second tile list over the same
    rows with tiles of that size, for a product that runs with another token tile (``linear(..., second_tiles=True)``)."""
    _i32(ids, "ids")
    _need(n_pairs <= layout.sorted_pair.numel(), "moe_sort: layout too small")
    if tile_m is not None:
        _need(tile_m >= layout.MIN_TILE, f"moe_sort: tiles of at least {layout.MIN_TILE} rows")
        layout.tile_m = tile_m
    _need(tile2_m == 0 or tile2_m >= layout.MIN_TILE, f"moe_sort: tiles of at least {layout.MIN_TILE} rows")
    layout.tile2_m = tile2_m
    code = _lib("moe_route").locus_moe_sort(
        _p(ids), I(n_pairs), I(layout.n_experts), I(layout.tile_m), _p(layout.counts),
        _p(layout.offsets), _p(layout.sorted_pair), _p(layout.pair_pos), _p(layout.tile_expert),
        _p(layout.tile_row0), _p(layout.tile_rows), _p(layout.n_tiles), I(tile2_m), _p(layout.tile2_expert),
        _p(layout.tile2_row0), _p(layout.tile2_rows), _p(layout.n_tiles2), _stream()
    )
    if code == 0 and layout.n_experts > MOE_SORT_ONE_LAUNCH_EXPERTS:
        _count_launches(1)
    _check(code, "moe_sort")


ROUTE_SMALL_PAIRS = 1024  # limits of the one-launch selection + layout
ROUTE_SMALL_EXPERTS = 512


def route_small_takes(n_tokens: int, top_k: int, n_experts: int) -> bool:
    """Whether ``route_small`` handles this batch (a decode-sized batch: its single block would be
    slow for more tokens)."""
    return n_tokens <= 16 and n_tokens * top_k <= ROUTE_SMALL_PAIRS and n_experts <= ROUTE_SMALL_EXPERTS


def route_small(logits: torch.Tensor, n_experts: int, has_gate: bool, ids: torch.Tensor, wts: torch.Tensor,
                gamma: Optional[torch.Tensor], layout: ExpertLayout, *, n_tokens: int, top_k: int, renorm: bool,
                scale: float = 1.0, tile_m: Optional[int] = None, score_fn: str = "softmax",
                sel_bias: Optional[torch.Tensor] = None, n_group: int = 1, n_group_used: int = 1,
                group_score: str = "top2") -> None:
    """``router_select`` followed by ``moe_sort`` in one launch, for batches that
    ``route_small_takes``: same picks, weights and layout."""
    _need(route_small_takes(n_tokens, top_k, n_experts), "route_small: batch too large")
    _need(logits.is_cuda and logits.dtype == torch.float32 and logits.stride(1) == 1, "route_small: float32 logits")
    _i32(ids, "ids")
    _need(wts.dtype == torch.float32 and wts.numel() >= n_tokens * top_k and ids.numel() >= n_tokens * top_k,
          "route_small: ids / wts too small")
    _need(n_tokens * top_k <= layout.sorted_pair.numel() and layout.n_experts == n_experts,
          "route_small: layout does not fit")
    if has_gate:
        _need(gamma is not None and gamma.dtype == torch.float32 and gamma.numel() >= n_tokens, "route_small: gamma")
    if tile_m is not None:
        _need(tile_m >= layout.MIN_TILE, f"route_small: tiles of at least {layout.MIN_TILE} rows")
        layout.tile_m = tile_m
    layout.tile2_m = 0  # this call writes the first tile list only: a second list of an earlier call is stale now
    code = _lib("moe_route").locus_route_small(
        _p(logits), I(logits.stride(0)), _p(ids), _p(wts), _p(gamma), I(n_tokens), I(n_experts), I(top_k),
        I(1 if has_gate else 0), I(1 if renorm else 0), F(scale),
        *_route_rule(score_fn, sel_bias, n_group, n_group_used, n_experts, "route_small", group_score), I(layout.tile_m), _p(layout.counts),
        _p(layout.offsets), _p(layout.sorted_pair), _p(layout.pair_pos), _p(layout.tile_expert),
        _p(layout.tile_row0), _p(layout.tile_rows), _p(layout.n_tiles), _stream()
    )
    _check(code, "route_small", f"(T={n_tokens}, E={n_experts}, k={top_k})")


def route_fused_small(h: torch.Tensor, w_all: torch.Tensor, logits: torch.Tensor, n_experts: int, has_gate: bool,
                      ids: torch.Tensor, wts: torch.Tensor, gamma: Optional[torch.Tensor], layout: ExpertLayout,
                      counter: torch.Tensor, *, n_tokens: int, top_k: int, renorm: bool, scale: float = 1.0,
                      tile_m: Optional[int] = None, score_fn: str = "softmax", sel_bias: Optional[torch.Tensor] = None,
                      n_group: int = 1, n_group_used: int = 1, logit_bias: Optional[torch.Tensor] = None,
                      group_score: str = "top2") -> None:
    """:func:`router_logits` (with ``logit_bias`` as its bias) followed by :func:`route_small` in ONE launch, for batches that ``route_small_takes``:
    the same logits (the same kernel computes them), picks, weights and layout.  ``counter``: one int32 that is
    zero before the call and zero after it."""
    _need(route_small_takes(n_tokens, top_k, n_experts), "route_fused_small: batch too large")
    _cuda_c(h, "h")
    _cuda_c(w_all, "w_all")
    T, H = n_tokens, h.shape[1]
    n = n_experts + (1 if has_gate else 0)
    _need(h.shape[0] >= T and w_all.shape[0] == n and w_all.shape[1] == H, "route_fused_small: shapes")
    _need(h.dtype == torch.bfloat16 and w_all.dtype == torch.bfloat16 and H % 8 == 0, "route_fused_small: bfloat16, H % 8 == 0")
    _need(logits.is_cuda and logits.dtype == torch.float32 and logits.shape[0] >= T and logits.shape[1] >= n
          and logits.stride(1) == 1, "route_fused_small: logits must be float32 [T, >= rows of w_all]")
    _i32(ids, "ids")
    _i32(counter, "counter")
    _need(wts.dtype == torch.float32 and wts.numel() >= T * top_k and ids.numel() >= T * top_k,
          "route_fused_small: ids / wts too small")
    _need(T * top_k <= layout.sorted_pair.numel() and layout.n_experts == n_experts, "route_fused_small: layout does not fit")
    if has_gate:
        _need(gamma is not None and gamma.dtype == torch.float32 and gamma.numel() >= T, "route_fused_small: gamma")
    if tile_m is not None:
        _need(tile_m >= layout.MIN_TILE, f"route_fused_small: tiles of at least {layout.MIN_TILE} rows")
        layout.tile_m = tile_m
    layout.tile2_m = 0  # as in route_small: no second tile list
    code = _lib("gemm_skinny").locus_router_fused_small(
        _p(h), _p(w_all), _p(logits), I(logits.stride(0)), _p(counter), _p(ids), _p(wts), _p(gamma), I(T), I(H),
        LL(h.stride(0)), I(n_experts), I(top_k), I(1 if has_gate else 0), I(1 if renorm else 0), F(scale),
        *_route_rule(score_fn, sel_bias, n_group, n_group_used, n_experts, "route_fused_small", group_score), I(layout.tile_m),
        _p(layout.counts), _p(layout.offsets), _p(layout.sorted_pair), _p(layout.pair_pos), _p(layout.tile_expert),
        _p(layout.tile_row0), _p(layout.tile_rows), _p(layout.n_tiles), _p(_logit_bias(logit_bias, n)), _stream()
    )
    _check(code, "route_fused_small", f"(T={T}, E={n_experts}, k={top_k})")


def moe_combine(x: torch.Tensor, pair_out: torch.Tensor, pair_pos: torch.Tensor, top_k: int) -> None:
    """x[t] += sum over slots (in slot order) of pair_out[pair_pos[t * k + slot]] (float32 or bfloat16 rows;
    the sum is float32)."""
    _cuda_c(x, "x")
    _cuda_c(pair_out, "pair_out")
    _i32(pair_pos, "pair_pos")
    T, H = x.shape
    _need(x.dtype == torch.float32 and pair_out.dtype in (torch.float32, torch.bfloat16),
          "moe_combine: float32 x, float32 or bfloat16 pair rows")
    _need(pair_out.shape[-1] == H, "moe_combine: width mismatch")
    code = _lib("elementwise").locus_moe_combine(_p(x), _p(pair_out), I(dtype_code(pair_out.dtype)), _p(pair_pos), I(T),
                                                 I(top_k), I(H), _stream())
    _check(code, "moe_combine")


def add_rows(x: torch.Tensor, y: torch.Tensor) -> None:
    """x += y, float32 rows of one shape."""
    _cuda_c(x, "x")
    _cuda_c(y, "y")
    _need(x.dtype == y.dtype == torch.float32 and x.shape == y.shape, "add_rows: float32 rows of one shape")
    code = _lib("elementwise").locus_add_rows(_p(x), _p(y), LL(x.numel()), _stream())
    _check(code, "add_rows")


def gather_rows(src: torch.Tensor, idx: torch.Tensor, div: int, out: torch.Tensor, n: int) -> None:
    """out[i] = src[idx[i] // div] for i < n."""
    _cuda_c(src, "src")
    _cuda_c(out, "out")
    _i32(idx, "idx")
    _need(src.dtype == out.dtype and src.shape[-1] == out.shape[-1], "gather_rows: mismatch")
    code = _lib("elementwise").locus_gather_rows(_p(src), I(dtype_code(src.dtype)), _p(idx), I(div), _p(out),
                                                 I(n), I(src.shape[-1]), _stream())
    _check(code, "gather_rows")


# ---------------------------------------------------------------------------
# sublayers that read the residual stream themselves and are normed on the way out
D = ctypes.c_double


def cast_rows(x: torch.Tensor, out: torch.Tensor) -> None:
    """out[i, :] = x[i, :] (float32 rows) in ``out``'s element type."""
    _cuda_c(x, "x")
    _cuda_c(out, "out")
    _need(x.dtype == torch.float32 and x.shape == out.shape, "cast_rows: float32 rows into rows of the same shape")
    code = _lib("elementwise").locus_cast_rows(_p(x), _p(out), I(dtype_code(out.dtype)), LL(x.numel()), _stream())
    _check(code, "cast_rows")


def rmsnorm_add(y: torch.Tensor, w: torch.Tensor, eps: float, x: torch.Tensor) -> None:
    """x[i] += y[i] * rsqrt(mean(y[i]^2) + eps) * w: the norm of a sublayer's output, added to the float32
    residual stream (statistics in float32)."""
    _cuda_c(y, "y")
    _cuda_c(w, "w")
    _cuda_c(x, "x")
    _need(y.dtype == torch.float32 and x.dtype == torch.float32 and y.shape == x.shape and w.numel() == y.shape[-1],
          "rmsnorm_add: float32 y and x of one shape, w of their width")
    code = _lib("elementwise").locus_rmsnorm_add(_p(y), _p(w), I(dtype_code(w.dtype)), F(eps), _p(x), I(y.shape[0]),
                                                 I(y.shape[-1]), _stream())
    _check(code, "rmsnorm_add")


# ---------------------------------------------------------------------------
# latent attention (csrc/latent_attention.cu)
LATENT_QUERY_TILE = 16   # queries per work item of latent_attn
LATENT_MAX_RANK = 512


def _freq(freq: Optional[torch.Tensor], rot_pairs: int, what: str) -> None:
    if rot_pairs > 0:
        _need(freq is not None and freq.is_cuda and freq.dtype == torch.float64 and freq.numel() >= rot_pairs,
              f"{what}: the frequencies must be float64 [rot_pairs] on the device")


def latent_prep(dqkv: torch.Tensor, positions: torch.Tensor, freq: Optional[torch.Tensor], magnitude: float,
                w_q: torch.Tensor, w_kv: torch.Tensor, eps: float, cq_out: torch.Tensor, pool: torch.Tensor,
                slots: torch.Tensor, *, q_rank: int, kv_rank: int, rot_dim: int, rot_pairs: int,
                write: bool = True, half_split: bool = False) -> None:
    """From the stacked down-projections ``dqkv`` [T, q_rank + kv_rank + rot_dim] (float32): the normed query
    latent into ``cq_out`` [T, q_rank]; the normed key/value latent and the rotated shared key part into the
    token's cache row (``pool`` [n_pages, 1, 1, page_tokens, kv_rank + rot_dim], ``slots[t]`` = page *
    page_tokens + offset).  Interleaved pairs (2i, 2i + 1), i < ``rot_pairs``, are turned by
    position * freq[i]; cosine and sine are multiplied by ``magnitude``.  ``half_split``: the pairs are (i, i +
    rot_pairs) instead.  ``q_rank`` 0: no query latent (``cq_out``, ``w_q`` None): the rows hold the key/value side alone."""
    _need(dqkv.is_cuda and dqkv.stride(1) == 1, "latent_prep: dqkv must be CUDA rows with unit stride")
    if q_rank > 0:
        _cuda_c(cq_out, "cq_out")
    _cuda_c(pool, "pool")
    _i32(positions, "positions")
    _i32(slots, "slots")
    T = dqkv.shape[0]
    _need(dqkv.dtype == torch.float32 and dqkv.shape[1] >= q_rank + (kv_rank + rot_dim if write else 0), "latent_prep: dqkv float32 of the stacked width")
    _need(q_rank == 0 or (cq_out.dtype == pool.dtype and cq_out.shape[0] >= T and cq_out.shape[1] == q_rank), "latent_prep: cq_out")
    _need(pool.shape[-1] == kv_rank + rot_dim and pool.shape[1] == 1 and pool.shape[2] == 1, "latent_prep: pool layout")
    _need(w_kv.numel() == kv_rank and w_kv.is_cuda and (q_rank == 0 or (w_q.dtype == w_kv.dtype and w_q.numel() == q_rank
                                                                     and w_q.is_cuda)), "latent_prep: norm weights")
    _need(positions.numel() >= T and slots.numel() >= T, "latent_prep: T mismatch")
    _freq(freq, rot_pairs, "latent_prep")
    code = _lib("latent_attention").locus_latent_prep(
        _p(dqkv), _p(positions), _p(freq), F(magnitude), _p(w_q if q_rank else None), _p(w_kv), I(dtype_code(w_kv.dtype)), F(eps),
        _p(cq_out if q_rank else None), _p(pool), I(dtype_code(pool.dtype)), _p(slots), I(T), I(q_rank), I(kv_rank), I(rot_dim),
        I(rot_pairs), I(1 if write else 0), I(1 if half_split else 0), I(dqkv.stride(0)), _stream())
    _check(code, "latent_prep")


def latent_q_split(q: torch.Tensor, positions: torch.Tensor, freq: Optional[torch.Tensor], magnitude: float,
                   q_nope_hm: torch.Tensor, q_rot: torch.Tensor, *, n_heads: int, nope_dim: int, rot_dim: int,
                   rot_pairs: int, half_split: bool = False) -> None:
    """``q`` [T, H * (nope_dim + rot_dim)], head by head [unrotated | rotated]: the unrotated parts go to
    ``q_nope_hm`` [H * T, nope_dim] (head-major: row h * T + t), the rotated parts, turned by the token's
    position, to ``q_rot`` [T, H * rot_dim]."""
    _cuda_c(q, "q")
    _cuda_c(q_nope_hm, "q_nope_hm")
    _cuda_c(q_rot, "q_rot")
    _i32(positions, "positions")
    T = q.shape[0]
    _need(q.shape[1] == n_heads * (nope_dim + rot_dim) and q.dtype == q_nope_hm.dtype == q_rot.dtype, "latent_q_split: q")
    _need(q_nope_hm.shape[0] >= n_heads * T and q_nope_hm.shape[1] == nope_dim, "latent_q_split: q_nope_hm")
    _need(q_rot.shape[0] >= T and q_rot.shape[1] == n_heads * rot_dim, "latent_q_split: q_rot")
    _freq(freq, rot_pairs, "latent_q_split")
    code = _lib("latent_attention").locus_latent_q_split(
        _p(q), I(dtype_code(q.dtype)), _p(positions), _p(freq), F(magnitude), _p(q_nope_hm), _p(q_rot), I(T),
        I(n_heads), I(nope_dim), I(rot_dim), I(rot_pairs), I(1 if half_split else 0), _stream())
    _check(code, "latent_q_split")


def latent_attn(q_abs_hm: torch.Tensor, q_rot: torch.Tensor, pool: torch.Tensor, sink: Optional[torch.Tensor],
                out_hm: torch.Tensor, *, seg_q0: torch.Tensor, seg_qn: torch.Tensor, seg_ctx: torch.Tensor,
                block_table: torch.Tensor, items: torch.Tensor, n_items: int, n_tokens: int, n_heads: int,
                kv_rank: int, rot_dim: int, page_tokens: int, window: int, scale: float) -> None:
    """Attention over latent cache rows [latent (kv_rank) | rotated key part (rot_dim)] that all heads share:
    score = (q_abs . latent + q_rot . key part) * scale over the keys a query sees (``window`` > 0: the last
    ``window`` positions, itself included), softmax whose denominator also holds exp(sink[h]) when ``sink`` is
    given, output = sum of p * latent.  ``q_abs_hm`` and ``out_hm`` are head-major [H * T, kv_rank]; ``items``
    [n_items, 2] = (segment, first query of a tile of ``LATENT_QUERY_TILE`` queries within it)."""
    _cuda_c(q_abs_hm, "q_abs_hm")
    _cuda_c(q_rot, "q_rot")
    _cuda_c(pool, "pool")
    _cuda_c(out_hm, "out_hm")
    _i32(block_table, "block_table")
    _i32(items, "items")
    T = n_tokens
    _need(q_abs_hm.dtype == q_rot.dtype == pool.dtype == out_hm.dtype, "latent_attn: one element type")
    _need(q_abs_hm.shape[0] >= n_heads * T and q_abs_hm.shape[1] == kv_rank and out_hm.shape[0] >= n_heads * T
          and out_hm.shape[1] == kv_rank and q_rot.shape[0] >= T and q_rot.shape[1] == n_heads * rot_dim,
          "latent_attn: shapes")
    _need(pool.shape[-1] == kv_rank + rot_dim and pool.shape[-2] == page_tokens, "latent_attn: pool layout")
    if sink is not None:
        _need(sink.is_cuda and sink.dtype == torch.float32 and sink.numel() == n_heads and sink.is_contiguous(),
              "latent_attn: sink must be float32 [H]")
    code = _lib("latent_attention").locus_latent_attn(
        _p(q_abs_hm), _p(q_rot), I(dtype_code(pool.dtype)), _p(pool), _p(sink), _p(out_hm), _p(seg_q0), _p(seg_qn),
        _p(seg_ctx), _p(block_table), I(block_table.shape[1]), _p(items), I(n_items), I(T), I(n_heads), I(kv_rank),
        I(rot_dim), I(page_tokens), I(window), F(scale), _stream())
    _check(code, "latent_attn", f"(heads {n_heads}, latent {kv_rank} + {rot_dim})")


# Long portions: the heads' keys and values of a segment's whole context are expanded into plain rows and the portion runs on
# the tcgen05 attention kernel.  A query-key pair then costs 2 x (key + value size) multiply-adds a head instead of 2 x 2 x rank
# on the mma.sync kernel (sizes of 128 on a latent of 512: a quarter, on the faster pipe); the expansion costs as much as that
# of two products per context row and is shared by the portion's queries.  Measured at 16 heads of 128 on a latent of 512, all
# kernels between the queries and the output projection, over the latents / expanded: 2,048 tokens 561 / 55 us; 128 tokens
# behind 0, 1,024 and 8,192 others 45 / 16, 77 / 34 and 307 / 91 us; 64 tokens over the latents 32, 54 and 157 us.
LATENT_EXPAND_FROM = 64          # new tokens of a segment from which on it is expanded
LATENT_EXPAND_ROWS = 16384       # most context rows of a step that are expanded ...
LATENT_EXPAND_BYTES = 512 << 20  # ... and most bytes of their keys and values; segments beyond run over the latents


def latent_expand_rows(dtype: torch.dtype, n_heads: int, nope_dim: int, rot_dim: int, v_dim: int, kv_rank: int) -> int:
    """Context rows of a step that may be expanded for the tcgen05 attention kernel; 0 where it does not take this mixer's sizes
    (bfloat16, keys without a rotated part and values of the kernel's head size)."""
    if not (USE_TENSOR_CORES and dtype == torch.bfloat16 and nope_dim == v_dim == TC_ATTN_HEAD_DIM and rot_dim == 0 and kv_rank % 8 == 0):
        return 0
    return min(LATENT_EXPAND_ROWS, LATENT_EXPAND_BYTES // (2 * n_heads * (nope_dim + v_dim)))


def latent_gather(pool: torch.Tensor, out: torch.Tensor, *, segs: torch.Tensor, n_segs: int, row0: torch.Tensor,
                  seg_qn: torch.Tensor, seg_ctx: torch.Tensor, block_table: torch.Tensor, page_tokens: int, longest: int) -> None:
    """out[row0[s] + t, :] = the leading elements of segment s's cache row of position t, for the ``n_segs`` segments that
    ``segs`` lists and all their positions (cached and new); ``longest``: the most positions of one of them."""
    _cuda_c(pool, "pool")
    _cuda_c(out, "out")
    for t, name in ((segs, "segs"), (row0, "row0"), (block_table, "block_table")):
        _i32(t, name)
    _need(pool.dtype == out.dtype and pool.shape[-2] == page_tokens and out.shape[1] <= pool.shape[-1] and pool.shape[1] == pool.shape[2] == 1,
          "latent_gather: rows of the pool's element type, at most as wide")
    code = _lib("latent_attention").locus_latent_gather(
        _p(pool), I(dtype_code(pool.dtype)), _p(out), _p(segs), I(n_segs), _p(row0), _p(seg_qn), _p(seg_ctx), _p(block_table),
        I(block_table.shape[1]), I(page_tokens), I(pool.shape[-1]), I(out.shape[1]), I(longest), _stream())
    _check(code, "latent_gather", f"(rows of {out.shape[1]} of {pool.shape[-1]})")


LATENT_MMA_RANKS = (32, 64, 96, 128, 160, 192, 224, 256, 320, 384, 448, 512)


def latent_attn_mma_takes(dtype: torch.dtype, kv_rank: int, rot_dim: int) -> bool:
    """Whether :func:`latent_attn_mma` takes this case: bfloat16, a latent whose size is a multiple of 32 up to 256 or of 64 up to 512, and a
    rotated part that is a multiple of 16 (or none); everything else runs on :func:`latent_attn`."""
    return (USE_TENSOR_CORES and dtype == torch.bfloat16 and kv_rank in LATENT_MMA_RANKS and rot_dim % 16 == 0)


def latent_mma_head_shift(n_heads: int) -> int:
    """log2 of the heads that share a block of :func:`latent_attn_mma` (its 64 rows are 64 >> shift queries times
    1 << shift heads): the smallest power of two that holds all heads, at most 16, so that a tile of keys in shared
    memory serves as many heads as possible and a block still holds several queries."""
    shift = 0
    while (1 << shift) < n_heads and shift < 4:
        shift += 1
    return shift


LATENT_MMA_MAX_SPLITS = 16


def latent_attn_mma_splits(n_items: int, n_heads: int, head_shift: int, max_keys: int) -> int:
    """Ranges the key tiles of every block of :func:`latent_attn_mma` are cut into: a step of single tokens (or of a
    short portion) behind long contexts makes a handful of blocks that would each walk all keys alone; then the keys
    are cut so that about every SM has a block, down to two tiles of 32 keys per range."""
    blocks = n_items * (-(-n_heads // (1 << head_shift)))
    tiles = -(-max_keys // 32)
    n_sm = _sm_count()
    if 2 * blocks > n_sm or tiles < 4:
        return 1
    return max(1, min(LATENT_MMA_MAX_SPLITS, n_sm // blocks, tiles // 2))


def latent_attn_mma_scratch(kv_rank: int) -> Tuple[int, int]:
    """Floats of the two scratch buffers (sums; maxima and denominators) for any cut that
    :func:`latent_attn_mma_splits` chooses: the ranges of a step never outnumber the SMs."""
    return _sm_count() * 64 * kv_rank, _sm_count() * 64 * 2


def latent_attn_mma(q_abs_hm: torch.Tensor, q_rot: torch.Tensor, pool: torch.Tensor, sink: Optional[torch.Tensor],
                    out_hm: torch.Tensor, *, seg_q0: torch.Tensor, seg_qn: torch.Tensor, seg_ctx: torch.Tensor,
                    block_table: torch.Tensor, items: torch.Tensor, n_items: int, n_tokens: int, n_heads: int,
                    kv_rank: int, rot_dim: int, page_tokens: int, window: int, scale: float, head_shift: int,
                    n_splits: int = 1, part_o: Optional[torch.Tensor] = None,
                    part_ml: Optional[torch.Tensor] = None) -> None:
    """:func:`latent_attn` on the tensor cores (bfloat16): same arguments and result, but ``items`` lists tiles of
    ``64 >> head_shift`` queries (:func:`latent_mma_head_shift`).  ``n_splits`` > 1
    (:func:`latent_attn_mma_splits`) with scratch of :func:`latent_attn_mma_scratch` floats: every block's keys are
    cut into that many ranges, merged in ascending order by a second kernel."""
    if n_splits > 1:
        units = n_items * (-(-n_heads // (1 << head_shift))) * n_splits
        _need(part_o is not None and part_ml is not None and part_o.dtype == part_ml.dtype == torch.float32
              and part_o.is_cuda and part_ml.is_cuda and part_o.numel() >= units * 64 * kv_rank
              and part_ml.numel() >= units * 128, "latent_attn_mma: scratch too small for these ranges")
    _cuda_c(q_abs_hm, "q_abs_hm")
    _cuda_c(q_rot, "q_rot")
    _cuda_c(pool, "pool")
    _cuda_c(out_hm, "out_hm")
    _i32(block_table, "block_table")
    _i32(items, "items")
    T = n_tokens
    _need(q_abs_hm.dtype == q_rot.dtype == pool.dtype == out_hm.dtype == torch.bfloat16, "latent_attn_mma: bfloat16 only")
    _need(q_abs_hm.shape[0] >= n_heads * T and q_abs_hm.shape[1] == kv_rank and out_hm.shape[0] >= n_heads * T
          and out_hm.shape[1] == kv_rank and q_rot.shape[0] >= T and q_rot.shape[1] == n_heads * rot_dim,
          "latent_attn_mma: shapes")
    _need(pool.shape[-1] == kv_rank + rot_dim and pool.shape[-2] == page_tokens, "latent_attn_mma: pool layout")
    if sink is not None:
        _need(sink.is_cuda and sink.dtype == torch.float32 and sink.numel() == n_heads and sink.is_contiguous(),
              "latent_attn_mma: sink must be float32 [H]")
    code = _lib("latent_attention").locus_latent_attn_mma(
        _p(q_abs_hm), _p(q_rot), _p(pool), _p(sink), _p(out_hm), _p(seg_q0), _p(seg_qn), _p(seg_ctx), _p(block_table),
        I(block_table.shape[1]), _p(items), I(n_items), I(T), I(n_heads), I(kv_rank), I(rot_dim), I(page_tokens),
        I(window), F(scale), I(head_shift), I(n_splits), _p(part_o if n_splits > 1 else None),
        _p(part_ml if n_splits > 1 else None), _stream())
    if n_splits > 1 and code == 0:
        _count_launches(1)
    _check(code, "latent_attn_mma", f"(heads {n_heads}, latent {kv_rank} + {rot_dim})")


LATENT_DECODE_RANKS, LATENT_DECODE_ROTS = (128, 256, 384, 512), (0, 32, 64)
LATENT_DECODE_HEADS, LATENT_DECODE_KEYS, LATENT_DECODE_MAX_RANGES = 16, 64, 64   # of a block; of a key tile


def latent_decode_takes(dtype: torch.dtype, kv_rank: int, rot_dim: int) -> bool:
    """Whether :func:`latent_decode` takes single tokens of this case; otherwise they run with the portions."""
    return USE_TENSOR_CORES and dtype == torch.bfloat16 and kv_rank in LATENT_DECODE_RANKS and rot_dim in LATENT_DECODE_ROTS


def latent_decode_ranges(n_items: int, n_heads: int, max_keys: int) -> int:
    """Ranges every request's key tiles are cut into: a block takes one, a block per SM, so the cut with the least rounds x
    (tiles of a range + what starting and merging one costs, in tiles), at most four blocks per SM (the scratch's size)."""
    n_sm = _sm_count()
    blocks = n_items * -(-n_heads // LATENT_DECODE_HEADS)
    tiles = -(-max_keys // LATENT_DECODE_KEYS)
    best, best_cost = 1, None
    for n in range(1, min(LATENT_DECODE_MAX_RANGES, tiles, max(1, 4 * n_sm // blocks)) + 1):
        cost = -(-blocks * n // n_sm) * (-(-tiles // n) + 2.0) + 0.05 * n
        if best_cost is None or cost < best_cost - 1e-9:
            best, best_cost = n, cost
    return best


def latent_decode_scratch(kv_rank: int) -> Tuple[int, int]:
    """Floats of the two scratch buffers for any cut that :func:`latent_decode_ranges` chooses."""
    units = 4 * _sm_count() * LATENT_DECODE_HEADS
    return units * kv_rank, units * 2


def latent_decode(q_abs_hm: torch.Tensor, q_rot: torch.Tensor, pool: torch.Tensor, sink: Optional[torch.Tensor],
                  out_hm: torch.Tensor, *, seg_q0: torch.Tensor, seg_ctx: torch.Tensor, block_table: torch.Tensor,
                  items: torch.Tensor, n_items: int, n_tokens: int, n_heads: int, kv_rank: int, rot_dim: int, page_tokens: int,
                  window: int, scale: float, n_ranges: int = 1, part_o: Optional[torch.Tensor] = None,
                  part_ml: Optional[torch.Tensor] = None) -> None:
    """:func:`latent_attn` of single new tokens: ``items`` [n_items] lists segments with one new token; every cached row is
    read once for sixteen heads.  ``n_ranges`` > 1 (:func:`latent_decode_ranges`) with scratch of
    :func:`latent_decode_scratch` floats: the keys of every request are cut into that many ranges, merged in ascending order."""
    _cuda_c(q_abs_hm, "q_abs_hm")
    _cuda_c(q_rot, "q_rot")
    _cuda_c(pool, "pool")
    _cuda_c(out_hm, "out_hm")
    _i32(block_table, "block_table")
    _i32(items, "items")
    T = n_tokens
    _need(q_abs_hm.dtype == q_rot.dtype == pool.dtype == out_hm.dtype == torch.bfloat16, "latent_decode: bfloat16 only")
    _need(q_abs_hm.shape[0] >= n_heads * T and q_abs_hm.shape[1] == kv_rank and out_hm.shape[0] >= n_heads * T
          and out_hm.shape[1] == kv_rank and q_rot.shape[0] >= T and q_rot.shape[1] == n_heads * rot_dim, "latent_decode: shapes")
    _need(pool.shape[-1] == kv_rank + rot_dim and pool.shape[-2] == page_tokens, "latent_decode: pool layout")
    if sink is not None:
        _need(sink.is_cuda and sink.dtype == torch.float32 and sink.numel() == n_heads and sink.is_contiguous(),
              "latent_decode: sink must be float32 [H]")
    if n_ranges > 1:
        units = n_items * -(-n_heads // LATENT_DECODE_HEADS) * n_ranges * LATENT_DECODE_HEADS
        _need(part_o is not None and part_ml is not None and part_o.is_cuda and part_ml.is_cuda
              and part_o.dtype == part_ml.dtype == torch.float32 and part_o.numel() >= units * kv_rank and part_ml.numel() >= 2 * units,
              "latent_decode: scratch too small for these ranges")
    code = _lib("latent_attention").locus_latent_decode(
        _p(q_abs_hm), _p(q_rot), _p(pool), _p(sink), _p(out_hm), _p(seg_q0), _p(seg_ctx), _p(block_table), I(block_table.shape[1]),
        _p(items), I(n_items), I(T), I(n_heads), I(kv_rank), I(rot_dim), I(page_tokens), I(window), F(scale), I(n_ranges),
        _p(part_o if n_ranges > 1 else None), _p(part_ml if n_ranges > 1 else None), _stream())
    if n_ranges > 1 and code == 0:
        _count_launches(1)
    _check(code, "latent_decode", f"(heads {n_heads}, latent {kv_rank} + {rot_dim}, {n_ranges} key ranges)")


def heads_to_rows(src_hm: torch.Tensor, out: torch.Tensor, *, n_tokens: int, n_heads: int) -> None:
    """``src_hm`` [H * T, d] head-major -> ``out`` [T, H * d]."""
    _cuda_c(src_hm, "src_hm")
    _cuda_c(out, "out")
    d = src_hm.shape[1]
    _need(src_hm.dtype == out.dtype and src_hm.shape[0] >= n_heads * n_tokens and out.shape[0] >= n_tokens
          and out.shape[1] == n_heads * d, "heads_to_rows: shapes")
    code = _lib("latent_attention").locus_heads_to_rows(_p(src_hm), I(dtype_code(out.dtype)), _p(out), I(n_tokens),
                                                        I(n_heads), I(d), _stream())
    _check(code, "heads_to_rows")


class HeadLayout:
    """The tile lists of a grouped product whose groups are the heads of a head-major tensor [H * T, ...]: head
    h owns the rows h * T .. (h + 1) * T.  It stands where :func:`linear` takes an :class:`ExpertLayout`; the lists
    themselves are device views that the step's plan wrote (parts.latent_attention.HeadTiles)."""

    def __init__(self, n_heads: int, tile_m: int, offsets, tile_expert, tile_row0, tile_rows, n_tiles,
                 max_tiles: int) -> None:
        self.n_experts, self.tile_m, self.tile2_m = n_heads, tile_m, 0
        self.offsets, self.tile_expert, self.tile_row0, self.tile_rows = offsets, tile_expert, tile_row0, tile_rows
        self.n_tiles, self.max_tiles = n_tiles, max_tiles

    def tiles_for(self, n_pairs: int, tile_m: Optional[int] = None) -> int:
        return self.max_tiles


def head_tile(n_tokens: int, dtype: torch.dtype, widths_ok: bool) -> int:
    """Row tile of the per-head products of ``n_tokens`` rows a head, by the kernel that :func:`linear` picks for
    it: 8 rows on the row-streaming kernels, 128 on the tcgen05 kernel, 64 on the CUDA cores."""
    if widths_ok and n_tokens <= FEW_ROWS:
        return FEW_ROWS
    if widths_ok and USE_TENSOR_CORES and dtype == torch.bfloat16:
        return 128
    return 64


# ---------------------------------------------------------------------------
# retention (csrc/retention.cu)
RETENTION_MAX_DIM = 256


RETENTION_CHUNK_FROM = 16   # segments with at least this many new tokens go to the chunked kernel


def retention_scan(qkvg: torch.Tensor, state: torch.Tensor, state_slots: torch.Tensor, seg_q0: torch.Tensor,
                   seg_qn: torch.Tensor, n_seg: int, decay: torch.Tensor, k_scale: float, o_raw: torch.Tensor, *,
                   n_heads: int, dim: int, v_dim: int, short: bool = True, long: bool = True,
                   longest_new: int = 0) -> None:
    """The recurrence S = decay[h] * S + (k * k_scale) v^T, o = S^T q over every segment's new tokens in order,
    from and into ``state`` [n_slots, H, dim, v_dim] (float32) of the segment's slot.  ``qkvg`` [T, >= 2 H dim +
    2 H v_dim] float32 with the columns [q | k | v | gate]; ``o_raw`` [T, H * v_dim] float32.

    Two kernels share the segments: those with fewer than ``RETENTION_CHUNK_FROM`` new tokens are walked token by
    token (a warp per few columns of the state), the longer ones chunk by chunk as small matrix products; ``short``
    / ``long`` say whether the step has segments of either kind at all (both True when the host cannot know);
    ``longest_new``: the most new tokens of a segment (0: the rows of ``qkvg``)."""
    _cuda_c(qkvg, "qkvg")
    _cuda_c(state, "state")
    _cuda_c(o_raw, "o_raw")
    _i32(state_slots, "state_slots")
    _need(qkvg.dtype == state.dtype == o_raw.dtype == decay.dtype == torch.float32, "retention_scan: float32 throughout")
    _need(tuple(state.shape[1:]) == (n_heads, dim, v_dim) and decay.numel() == n_heads and decay.is_cuda,
          "retention_scan: state [slots, H, dim, v_dim], decay [H]")
    _need(o_raw.shape[1] == n_heads * v_dim and o_raw.shape[0] >= qkvg.shape[0], "retention_scan: o_raw")
    if short:
        code = _lib("retention").locus_retention_scan(
            _p(qkvg), I(qkvg.stride(0)), _p(state), _p(state_slots), _p(seg_q0), _p(seg_qn), I(n_seg), _p(decay),
            F(k_scale), _p(o_raw), I(n_heads), I(dim), I(v_dim), I(RETENTION_CHUNK_FROM if long else 0), _stream())
        _check(code, "retention_scan", f"(heads {n_heads}, dim {dim}, v_dim {v_dim})")
    if long:
        code = _lib("retention").locus_retention_chunked(
            _p(qkvg), I(qkvg.stride(0)), _p(state), _p(state_slots), _p(seg_q0), _p(seg_qn), I(n_seg), _p(decay),
            F(k_scale), _p(o_raw), I(n_heads), I(dim), I(v_dim), I(RETENTION_CHUNK_FROM if short else 1),
            I(longest_new or qkvg.shape[0]), _stream())
        if code == 0:
            _count_launches(1)   # two kernels: the chunks' own terms, then the walk over the chunks
        _check(code, "retention_chunked", f"(heads {n_heads}, dim {dim}, v_dim {v_dim})")


def retention_gate_norm(o_raw: torch.Tensor, qkvg: torch.Tensor, gate_offset: int, eps: float, out: torch.Tensor, *,
                        n_heads: int, v_dim: int) -> None:
    """out[t, h, :] = o_raw[t, h, :] / rms(o_raw[t, h, :]) * silu(gate[t, h, :]), the gate being the columns of
    ``qkvg`` from ``gate_offset`` on."""
    _cuda_c(o_raw, "o_raw")
    _cuda_c(qkvg, "qkvg")
    _cuda_c(out, "out")
    T = out.shape[0]
    _need(o_raw.dtype == qkvg.dtype == torch.float32 and o_raw.shape[0] >= T and qkvg.shape[0] >= T
          and o_raw.shape[1] == out.shape[1] == n_heads * v_dim and qkvg.shape[1] >= gate_offset + n_heads * v_dim,
          "retention_gate_norm: shapes")
    code = _lib("retention").locus_retention_gate_norm(_p(o_raw), _p(qkvg), I(qkvg.stride(0)), I(gate_offset), F(eps),
                                                       _p(out), I(dtype_code(out.dtype)), I(T), I(n_heads), I(v_dim),
                                                       _stream())
    _check(code, "retention_gate_norm")


# ---------------------------------------------------------------------------
# several copies of the residual stream, layer norm

MAX_STREAMS = 8


def layernorm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float, out: torch.Tensor,
              rows: Optional[torch.Tensor] = None, n_streams: int = 1, coef: Optional[torch.Tensor] = None) -> None:
    """out[i] = layer norm (weight ``w``, bias ``b``; mean and variance in float32) of u = sum_s coef[s] * x[r, s, :],
    r = rows[i] if ``rows`` else i.  ``x`` [n, n_streams * H] float32 holds ``n_streams`` copies of the residual stream
    per row; ``coef`` [n_streams] float32, None: the plain sum (with one stream: the row itself)."""
    _cuda_c(x, "x")
    _cuda_c(out, "out")
    n, H = out.shape
    _need(x.dtype == torch.float32 and x.shape[1] == n_streams * H and 1 <= n_streams <= MAX_STREAMS,
          "layernorm: x must be float32 [n, n_streams * H]")
    _need(w.numel() == H and b.numel() == H and w.dtype == b.dtype and w.is_cuda and b.is_cuda, "layernorm: w, b [H]")
    if coef is not None:
        _need(coef.is_cuda and coef.dtype == torch.float32 and coef.numel() == n_streams, "layernorm: coef [n_streams] float32")
    if rows is not None:
        _i32(rows, "rows")
        _need(rows.numel() == n, "layernorm: rows/out mismatch")
    else:
        _need(x.shape[0] >= n, "layernorm: x/out mismatch")
    code = _lib("elementwise").locus_layernorm(_p(x), I(n_streams), _p(coef), _p(w), _p(b), I(dtype_code(w.dtype)), F(eps),
                                               _p(out), I(dtype_code(out.dtype)), _p(rows), I(n), I(H), _stream())
    _check(code, "layernorm")


def stream_update(x: torch.Tensor, y: torch.Tensor, mix: torch.Tensor, out_coef: torch.Tensor, n_streams: int) -> None:
    """x[r, t, :] <- sum_s mix[s, t] * x[r, s, :] + out_coef[t] * y[r, :] for the rows of ``y``, every copy t at once
    from the old copies.  ``x`` [>= n, n_streams * H] and ``y`` [n, H] float32; ``mix`` [n_streams, n_streams] (indexed
    [from, to]) and ``out_coef`` [n_streams] float32."""
    _cuda_c(x, "x")
    _cuda_c(y, "y")
    n, H = y.shape
    _need(x.dtype == y.dtype == torch.float32 and x.shape[0] >= n and x.shape[1] == n_streams * H
          and 1 <= n_streams <= MAX_STREAMS, "stream_update: x [n, n_streams * H], y [n, H] float32")
    _need(mix.is_cuda and out_coef.is_cuda and mix.dtype == out_coef.dtype == torch.float32
          and mix.numel() == n_streams * n_streams and out_coef.numel() == n_streams and mix.is_contiguous(),
          "stream_update: mix [S, S], out_coef [S] float32")
    code = _lib("elementwise").locus_stream_update(_p(x), _p(y), _p(mix), _p(out_coef), I(n_streams), I(n), I(H), _stream())
    _check(code, "stream_update")


def moe_identity(h: torch.Tensor, wts: torch.Tensor, layout: ExpertLayout, pair_out: torch.Tensor, *, n_pairs: int,
                 top_k: int, n_real: int) -> None:
    """Experts from ``n_real`` on have no weights and pass their input through: their tiles are taken off the layout's
    tile lists and their rows are written, pair_out[r] = wts[pair] * h[pair // top_k] for the layout's rows r of
    those experts.  To be called behind the call that filled the layout and before the grouped products."""
    _cuda_c(h, "h")
    _cuda_c(pair_out, "pair_out")
    H = h.shape[1]
    _need(wts.dtype == torch.float32 and wts.numel() >= n_pairs and pair_out.shape[0] >= n_pairs
          and pair_out.shape[1] == H and 0 <= n_real <= layout.n_experts, "moe_identity: shapes")
    second = layout.tile2_m > 0
    code = _lib("moe_route").locus_moe_identity(
        _p(h), I(dtype_code(h.dtype)), _p(wts), _p(layout.offsets), _p(layout.sorted_pair), _p(pair_out),
        I(dtype_code(pair_out.dtype)), I(n_pairs), I(top_k), I(H), I(n_real), _p(layout.tile_expert), _p(layout.n_tiles),
        _p(layout.tile2_expert if second else None), _p(layout.n_tiles2 if second else None), I(layout.max_tiles),
        _stream())
    _check(code, "moe_identity")


# ---------------------------------------------------------------------------
# gated linear recurrence and the mixers around it

RECURRENCE_MAX_DIM = 256
RECURRENCE_CHUNK_FROM = 16   # segments with at least this many new tokens go to the chunked kernels


def _f32c(t: torch.Tensor, name: str) -> None:
    _need(t.is_cuda and t.dtype == torch.float32 and t.stride(-1) == 1, f"{name} must be a float32 CUDA tensor with unit stride")


def gated_recurrence(q: torch.Tensor, off_q: int, k: torch.Tensor, off_k: int, v: torch.Tensor, off_v: int,
                     keep: torch.Tensor, take: torch.Tensor, state: torch.Tensor, state_offset: int,
                     state_slots: torch.Tensor, seg_q0: torch.Tensor, seg_qn: torch.Tensor, n_seg: int, out: torch.Tensor,
                     *, n_heads: int, heads_per_group: int, dim: int, v_dim: int, ones: bool = False,
                     q_scale: float = 1.0, short: bool = True, long: bool = True, longest_new: int = 0) -> None:
    """S = keep[t, h] * S + take[t, h] * k v^T, o = S^T (q * q_scale) per request and head over every segment's new
    tokens in order, from and into the request's state slot.  ``q``, ``k``, ``v``: float32 row matrices [T, .] in which
    head h's q and k start at column ``off_q`` / ``off_k`` + (h // heads_per_group) * dim and its v at ``off_v`` + h *
    v_dim.  ``keep``, ``take`` [T, n_heads] float32.  ``state`` [n_slots, floats per slot] float32: head h's matrix
    [dim, v_dim (+1)] starts ``state_offset`` + h * dim * (v_dim (+1)) floats into a slot.  ``ones``: the state has one
    column more, whose v is 1 (the recurrence of k alone); ``out`` [T, n_heads * (v_dim (+1))] float32.

    Segments with fewer than ``RECURRENCE_CHUNK_FROM`` new tokens are walked token by token, longer ones chunk by chunk
    as small matrix products; ``short`` / ``long`` say whether the step has segments of either kind (both True when the
    host cannot know); ``longest_new``: the most new tokens of a segment (0: the rows of ``out``)."""
    for t, name in ((q, "q"), (k, "k"), (v, "v"), (keep, "keep"), (take, "take"), (out, "out")):
        _f32c(t, f"gated_recurrence: {name}")
    _cuda_c(state, "state")
    _i32(state_slots, "state_slots")
    dvx = v_dim + (1 if ones else 0)
    _need(state.dtype == torch.float32 and state.dim() == 2
          and state_offset + n_heads * dim * dvx <= state.shape[1], "gated_recurrence: the state does not hold the heads")
    _need(keep.shape[1] == n_heads and take.shape[1] == n_heads and keep.is_contiguous() and take.is_contiguous(),
          "gated_recurrence: keep, take [T, n_heads]")
    _need(out.shape[1] == n_heads * dvx and out.is_contiguous(), "gated_recurrence: out [T, n_heads * columns]")
    _need(dim <= RECURRENCE_MAX_DIM, f"gated_recurrence: dim {dim} exceeds {RECURRENCE_MAX_DIM}")
    args = (_p(q), I(q.stride(0)), I(off_q), _p(k), I(k.stride(0)), I(off_k), _p(v), I(v.stride(0)), I(off_v), _p(keep),
            _p(take), ctypes.c_void_p(state.data_ptr() + 4 * state_offset), LL(state.stride(0)), _p(state_slots),
            _p(seg_q0), _p(seg_qn), I(n_seg), F(q_scale), _p(out), I(out.stride(0)), I(n_heads), I(heads_per_group),
            I(dim), I(v_dim), I(1 if ones else 0))
    what = f"(heads {n_heads}, dim {dim}, v_dim {v_dim})"
    if short:
        code = _lib("recurrence").locus_gated_scan(*args, I(RECURRENCE_CHUNK_FROM if long else 0), _stream())
        _check(code, "gated_scan", what)
    if long:
        code = _lib("recurrence").locus_gated_chunked(*args, I(RECURRENCE_CHUNK_FROM if short else 1),
                                                      I(longest_new or out.shape[0]), _stream())
        if code == 0:
            _count_launches(1)   # two kernels: the chunks' own terms, then the walk over the chunks
        _check(code, "gated_chunked", what)


def mlstm_gates(proj: torch.Tensor, off_i: int, off_f: int, cap: float, state: torch.Tensor, m_offset: int,
                state_slots: torch.Tensor, seg_q0: torch.Tensor, seg_qn: torch.Tensor, n_seg: int, keep: torch.Tensor,
                take: torch.Tensor, m_out: torch.Tensor, *, n_heads: int) -> None:
    """From the pre-activations in columns ``off_i`` + h and ``off_f`` + h of ``proj`` (float32 rows): i = cap *
    tanh(z_i / cap), f = logsigmoid(cap * tanh(z_f / cap)), the running maximum m_t = max(f + m_(t-1), i) (carried in
    the state slot at ``m_offset`` + h), keep = exp(f + m_(t-1) - m_t), take = exp(i - m_t); ``m_out`` gets m_t.  All
    [T, n_heads] float32."""
    _f32c(proj, "mlstm_gates: proj")
    _cuda_c(state, "state")
    for t in (keep, take, m_out):
        _need(t.is_cuda and t.dtype == torch.float32 and t.is_contiguous() and t.shape[1] == n_heads, "mlstm_gates: [T, n_heads] float32")
    _need(state.dtype == torch.float32 and state.dim() == 2 and m_offset + n_heads <= state.shape[1], "mlstm_gates: state")
    code = _lib("mlstm").locus_mlstm_gates(_p(proj), I(proj.stride(0)), I(off_i), I(off_f), F(cap),
                                           ctypes.c_void_p(state.data_ptr() + 4 * m_offset), LL(state.stride(0)),
                                           _p(state_slots), _p(seg_q0), _p(seg_qn), I(n_seg), _p(keep), _p(take), _p(m_out),
                                           I(n_heads), _stream())
    _check(code, "mlstm_gates")


def mlstm_out(o_raw: torch.Tensor, m_t: torch.Tensor, proj: torch.Tensor, off_g: int, w: torch.Tensor, eps: float,
              out: torch.Tensor, *, n_heads: int, v_dim: int) -> None:
    """o_raw [T, n_heads * (v_dim + 1)]: per head the numerator and, behind it, n . q.  out[t, h, :] = (numerator /
    (max(|n . q|, exp(-m_t)) + 1e-6)) / its root mean square * w[h, :] * sigmoid(gate), the gate being the columns of
    ``proj`` from ``off_g`` on."""
    _f32c(o_raw, "mlstm_out: o_raw")
    _f32c(proj, "mlstm_out: proj")
    _cuda_c(out, "out")
    T = out.shape[0]
    _need(o_raw.is_contiguous() and o_raw.shape[1] == n_heads * (v_dim + 1) and out.shape[1] == n_heads * v_dim
          and w.numel() == n_heads * v_dim and m_t.dtype == torch.float32 and m_t.is_contiguous(), "mlstm_out: shapes")
    code = _lib("mlstm").locus_mlstm_out(_p(o_raw), _p(m_t), _p(proj), I(proj.stride(0)), I(off_g), _p(w),
                                         I(dtype_code(w.dtype)), F(eps), _p(out), I(dtype_code(out.dtype)), I(T),
                                         I(n_heads), I(v_dim), _stream())
    _check(code, "mlstm_out")


SSM_MAX_TAPS = 16


def ssm_conv(proj: torch.Tensor, off_xbc: int, off_dt: int, conv_w: torch.Tensor, conv_b: torch.Tensor,
             dt_bias: torch.Tensor, a_log: torch.Tensor, state: torch.Tensor, conv_offset: int,
             state_slots: torch.Tensor, seg_q0: torch.Tensor, seg_qn: torch.Tensor, n_seg: int, act: torch.Tensor,
             keep: torch.Tensor, take: torch.Tensor, *, n_heads: int, longest_new: int = 0) -> None:
    """act[t, c] = silu(conv_b[c] + sum_j conv_w[c, j] * input(t - (taps - 1) + j, c)), the inputs being the columns of
    ``proj`` from ``off_xbc`` on and, before a portion's first token, the ``taps`` - 1 inputs that the request's
    state slot holds ([channels, taps - 1] floats from ``conv_offset`` on; they move on by the portion's tokens in the
    same call).  Also dt = softplus(proj[t, off_dt + h] + dt_bias[h]), keep = exp(-exp(a_log[h]) * dt), take = dt."""
    _f32c(proj, "ssm_conv: proj")
    _cuda_c(state, "state")
    channels, taps = conv_w.shape
    _need(conv_w.is_contiguous() and conv_b.numel() == channels and conv_w.dtype == conv_b.dtype and 1 <= taps <= SSM_MAX_TAPS,
          "ssm_conv: conv weights [channels, taps], bias [channels]")
    _need(dt_bias.numel() == n_heads and a_log.numel() == n_heads and dt_bias.dtype == a_log.dtype, "ssm_conv: dt_bias, A_log [heads]")
    _need(state.dtype == torch.float32 and state.dim() == 2 and conv_offset + channels * (taps - 1) <= state.shape[1], "ssm_conv: state")
    for t, wdt in ((act, channels), (keep, n_heads), (take, n_heads)):
        _need(t.is_cuda and t.dtype == torch.float32 and t.is_contiguous() and t.shape[1] == wdt, "ssm_conv: outputs")
    code = _lib("state_space").locus_ssm_conv(
        _p(proj), I(proj.stride(0)), I(off_xbc), I(off_dt), _p(conv_w), _p(conv_b), I(dtype_code(conv_w.dtype)),
        _p(dt_bias), _p(a_log), I(dtype_code(a_log.dtype)), ctypes.c_void_p(state.data_ptr() + 4 * conv_offset),
        LL(state.stride(0)), _p(state_slots), _p(seg_q0), _p(seg_qn), I(n_seg), I(longest_new or act.shape[0]), _p(act),
        _p(keep), _p(take), I(channels), I(taps), I(n_heads), _stream())
    if code == 0 and taps > 1:
        _count_launches(1)
    _check(code, "ssm_conv")


def ssm_out(y: torch.Tensor, act: torch.Tensor, proj: torch.Tensor, off_z: int, d_skip: torch.Tensor, w: torch.Tensor,
            eps: float, out: torch.Tensor, *, parts: int, v_dim: int) -> None:
    """out[t] = ((y[t] + d_skip[head] * x[t]) * silu(z[t])), each of ``parts`` equal parts of the row divided by its
    root mean square, times ``w``; x: the first columns of ``act``, z: the columns of ``proj`` from ``off_z`` on."""
    _f32c(y, "ssm_out: y")
    _f32c(act, "ssm_out: act")
    _f32c(proj, "ssm_out: proj")
    _cuda_c(out, "out")
    T, inner = out.shape
    _need(y.is_contiguous() and act.is_contiguous() and y.shape[1] == inner and act.shape[1] >= inner
          and w.numel() == inner and d_skip.numel() * v_dim == inner and inner % parts == 0, "ssm_out: shapes")
    code = _lib("state_space").locus_ssm_out(_p(y), _p(act), I(act.shape[1]), _p(proj), I(proj.stride(0)), I(off_z),
                                             _p(d_skip), I(dtype_code(d_skip.dtype)), _p(w), I(dtype_code(w.dtype)), F(eps),
                                             _p(out), I(dtype_code(out.dtype)), I(T), I(parts), I(inner), I(v_dim), _stream())
    _check(code, "ssm_out")


# ---------------------------------------------------------------------------
# between a stacked projection and its attention or recurrence (csrc/short_conv.cu), the gated delta rule
# (csrc/delta_rule.cu)

PREP_MAX_TAPS = 16
PREP_MAX_DIM = 256
HEAD_NORMS = {None: 0, "rms": 1, "unit": 2, "head": 3}


def head_prep(proj: torch.Tensor, *, offsets, heads, dims, laid, state_slots: torch.Tensor, seg_q0: torch.Tensor,
              seg_qn: torch.Tensor, n_seg: int, longest_new: int, positions: torch.Tensor, q_out: torch.Tensor,
              k_out: Optional[torch.Tensor] = None, v_out: Optional[torch.Tensor] = None,
              pool: Optional[torch.Tensor] = None, slots: Optional[torch.Tensor] = None, page_tokens: int = 0,
              write_kv: bool = True, conv: Optional[torch.Tensor] = None, state: Optional[torch.Tensor] = None,
              conv_offset: int = 0, move_state: bool = True, act: bool = False,
              inv_freq: Optional[torch.Tensor] = None, rot: int = 0, norm: Optional[str] = None, eps: float = 0.0,
              q_scale: float = 1.0, gates=None, interleaved: bool = False, norm_weights=None,
              n_rows: int = 0, q_temp=None) -> None:
    """From the float32 rows ``proj`` of a stacked projection to q in rows and k, v in rows or cache pages, in one
    launch.  ``offsets``, ``heads``, ``dims``, ``laid``: for q, k, v the first column in ``proj``, the number of heads,
    the per-head size and the size a head is laid out at in the output (zeros behind its own elements).  In this
    order, each only if given: ``conv`` [channels, taps] (the channels of q, k, v one behind the other), a causal
    convolution over time per channel, y_t = sum_j conv[c, j] u_(t - taps + 1 + j), whose inputs before a portion's
    first token come from the request's slot of ``state`` ([channels, taps - 1] floats from ``conv_offset`` on;
    moved on by the portion's tokens in the same call unless ``move_state`` is off); ``act``: silu; ``inv_freq``
    [rot / 2]: q's and k's pairs (i, i + rot / 2) rotated by position * inv_freq[i]; ``norm`` "rms": q and k divided
    by sqrt(mean(x^2) + eps) per head, "unit": by sqrt(sum(x^2) + eps), "head": by sqrt(mean(x^2) + eps) and multiplied by
    ``norm_weights`` = (q's, k's) [dim] in FRONT of the rotation; ``interleaved``: the rotation takes the pairs (2i, 2i + 1)
    instead; ``n_rows`` > 0: the segments' rows are the rows 0 .. n_rows - 1 of ``proj`` without a gap (the kernel of a block
    per token then runs where it can); ``q_scale`` on q; ``q_temp`` = (coef, every): q also
    multiplied by 1 + coef * ln(floor((p + 1) / every) + 1) at position p.  ``offsets`` may name one stretch twice (values that
    are the keys as projected).  The outputs share one
    element type; with ``pool`` (a layer's pages [n_pages, 2, heads_k, page_tokens, laid]) k and v go to ``slots``.
    ``gates`` = (beta, decay, off_b, off_a, a_log, dt_bias): also beta = sigmoid(proj[:, off_b + h]) and decay =
    exp(-exp(a_log[h]) * softplus(proj[:, off_a + h] + dt_bias[h])), [T, heads] float32 each."""
    _f32c(proj, "head_prep: proj")
    _cuda_c(q_out, "q_out")
    _i32(positions, "positions")
    sizes = (ctypes.c_int * 12)(*[int(v) for v in (*offsets, *heads, *dims, *laid)])
    out_dt = q_out.dtype
    _need(q_out.shape[1] == heads[0] * laid[0] and q_out.shape[0] >= n_rows and proj.shape[0] >= n_rows, "head_prep: q_out width")
    if pool is not None:
        _cuda_c(pool, "pool")
        _i32(slots, "slots")
        _need(pool.dtype == out_dt and tuple(pool.shape[1:]) == (2, heads[1], page_tokens, laid[1]) and laid[1] == laid[2],
              "head_prep: pool layout")
    elif heads[1] or heads[2]:
        for t, w in ((k_out, 1), (v_out, 2)):
            _need(t is not None and t.is_cuda and t.is_contiguous() and t.dtype == out_dt and t.shape[1] == heads[w] * laid[w],
                  "head_prep: k_out, v_out rows")
    taps = 1
    state_ptr, stride = None, 0
    if conv is not None:
        _cuda_c(conv, "conv")
        channels = sum(h * d for h, d in zip(heads, dims))
        taps = conv.shape[1]
        _need(conv.shape[0] == channels and 1 <= taps <= PREP_MAX_TAPS, "head_prep: conv [channels, taps]")
        if taps > 1:
            _need(state is not None and state.is_cuda and state.dtype == torch.float32 and state.dim() == 2
                  and state.stride(1) == 1 and conv_offset + channels * (taps - 1) <= state.shape[1], "head_prep: state")
            state_ptr, stride = ctypes.c_void_p(state.data_ptr() + 4 * conv_offset), state.stride(0)
    if inv_freq is not None:
        _need(inv_freq.dtype == torch.float32 and inv_freq.is_cuda and inv_freq.numel() == rot // 2, "head_prep: inv_freq [rot / 2]")
    q_w, k_w = norm_weights if norm_weights is not None else (None, None)
    _need((norm == "head") == (q_w is not None), "head_prep: norm_weights go with the norm 'head'")
    _need(q_temp is None or q_temp[1] > 0, "head_prep: q_temp (coef, every) needs a positive every")
    for t, which in ((q_w, 0), (k_w, 1)):
        _need(t is None or (t.is_cuda and t.is_contiguous() and t.numel() == dims[which] and t.dtype == q_w.dtype), "head_prep: norm_weights [dim]")
    beta = decay = a_log = dt_bias = None
    off_b = off_a = gate_heads = gate_dt = 0
    if gates is not None:
        beta, decay, off_b, off_a, a_log, dt_bias = gates
        gate_heads = beta.shape[1]
        _need(beta.dtype == decay.dtype == torch.float32 and beta.is_contiguous() and decay.is_contiguous()
              and decay.shape[1] == gate_heads and a_log.numel() == gate_heads and dt_bias.numel() == gate_heads
              and a_log.dtype == dt_bias.dtype, "head_prep: gates")
        gate_dt = dtype_code(a_log.dtype)
    code = _lib("short_conv").locus_head_prep(
        _p(proj), I(proj.stride(0)), sizes, _p(conv), I(dtype_code(conv.dtype) if conv is not None else 0), I(taps),
        I(1 if act else 0), state_ptr, LL(stride), I(1 if move_state else 0), _p(state_slots), _p(seg_q0), _p(seg_qn),
        I(n_seg), I(longest_new), I(n_rows), _p(positions), _p(inv_freq), I(rot if inv_freq is not None else 0),
        I(1 if interleaved else 0), I(HEAD_NORMS[norm]), _p(q_w), _p(k_w), I(dtype_code(q_w.dtype) if q_w is not None else 0),
        F(eps), F(q_scale), F(q_temp[0] if q_temp else 0.0), D(q_temp[1] if q_temp else 1.0), _p(q_out), _p(k_out), _p(v_out), _p(pool), _p(slots), I(page_tokens), I(1 if write_kv else 0),
        I(dtype_code(out_dt)), _p(beta), _p(decay), I(off_b), I(off_a), I(gate_heads), _p(a_log), _p(dt_bias), I(gate_dt),
        _stream())
    if code == 0 and conv is not None and taps > 1 and move_state and n_seg > 0 and longest_new > 0:
        _count_launches(1)
    _check(code, "head_prep")


def gate_rows(o: torch.Tensor, proj: torch.Tensor, off: int, *, n_heads: int, dim: int, laid: int) -> None:
    """o[t, h, :dim] *= sigmoid(proj[t, off + h * dim + .]) in place; o's heads are laid out at ``laid`` elements."""
    _cuda_c(o, "o")
    _f32c(proj, "gate_rows: proj")
    _need(o.shape[1] == n_heads * laid and proj.shape[1] >= off + n_heads * dim and proj.shape[0] >= o.shape[0], "gate_rows: shapes")
    code = _lib("short_conv").locus_gate_rows(_p(o), I(dtype_code(o.dtype)), I(o.stride(0)), _p(proj), I(proj.stride(0)),
                                              I(off), I(n_heads * dim), I(dim), I(laid), I(o.shape[0]), _stream())
    _check(code, "gate_rows")


DELTA_MAX_DIM = 256


def delta_rule(q: torch.Tensor, off_q: int, k: torch.Tensor, off_k: int, v: torch.Tensor, off_v: int, beta: torch.Tensor,
               decay: torch.Tensor, state: torch.Tensor, state_offset: int, state_slots: torch.Tensor, seg_q0: torch.Tensor,
               seg_qn: torch.Tensor, n_seg: int, out: torch.Tensor, *, n_heads: int, heads_per_group: int, dim: int,
               v_dim: int) -> None:
    """The gated delta rule per request and head over every segment's new tokens in order, from and into the request's
    state slot: S <- decay S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q.  ``q``, ``k``, ``v``: float32 row matrices
    in which head h's q and k start at column ``off_q`` / ``off_k`` + (h // heads_per_group) * dim and its v at
    ``off_v`` + h * v_dim; ``beta``, ``decay`` [T, n_heads] float32; head h's state [dim, v_dim] starts ``state_offset``
    + h * dim * v_dim floats into a slot of ``state`` [n_slots, floats]; ``out`` [T, n_heads * v_dim] float32."""
    for t, name in ((q, "q"), (k, "k"), (v, "v"), (beta, "beta"), (decay, "decay"), (out, "out")):
        _f32c(t, f"delta_rule: {name}")
    _i32(state_slots, "state_slots")
    _need(state.is_cuda and state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1
          and state_offset + n_heads * dim * v_dim <= state.shape[1], "delta_rule: the state does not hold the heads")
    _need(beta.shape[1] == n_heads and decay.shape[1] == n_heads and beta.is_contiguous() and decay.is_contiguous(),
          "delta_rule: beta, decay [T, n_heads]")
    _need(out.shape[1] == n_heads * v_dim and dim <= DELTA_MAX_DIM, "delta_rule: out [T, n_heads * v_dim], dim <= 256")
    code = _lib("delta_rule").locus_delta_scan(
        _p(q), I(q.stride(0)), I(off_q), _p(k), I(k.stride(0)), I(off_k), _p(v), I(v.stride(0)), I(off_v), _p(beta),
        _p(decay), ctypes.c_void_p(state.data_ptr() + 4 * state_offset), LL(state.stride(0)), _p(state_slots), _p(seg_q0),
        _p(seg_qn), I(n_seg), _p(out), I(out.stride(0)), I(n_heads), I(heads_per_group), I(dim), I(v_dim), _stream())
    _check(code, "delta_scan", f"(heads {n_heads}, dim {dim}, v_dim {v_dim})")


def delta_out(o: torch.Tensor, proj: torch.Tensor, off_g: int, w: torch.Tensor, eps: float, out: torch.Tensor, *,
              n_heads: int, v_dim: int) -> None:
    """out[t, h, :] = o[t, h, :] / sqrt(mean(o[t, h, :]^2) + eps) * w * silu(gate[t, h, :]); the gate: the columns of
    ``proj`` from ``off_g`` on; ``w`` [v_dim] (one weight for every head) or [n_heads * v_dim]."""
    _f32c(o, "delta_out: o")
    _f32c(proj, "delta_out: proj")
    _cuda_c(out, "out")
    _cuda_c(w, "w")
    T = out.shape[0]
    _need(o.is_contiguous() and o.shape[1] == out.shape[1] == n_heads * v_dim and w.numel() in (v_dim, n_heads * v_dim)
          and proj.shape[1] >= off_g + n_heads * v_dim, "delta_out: shapes")
    code = _lib("delta_rule").locus_delta_out(_p(o), _p(proj), I(proj.stride(0)), I(off_g), _p(w), I(dtype_code(w.dtype)),
                                              I(w.numel()), F(eps), _p(out), I(dtype_code(out.dtype)), I(T), I(n_heads),
                                              I(v_dim), _stream())
    _check(code, "delta_out")



# ---------------------------------------------------------------------------
# an embedding with a hashed pair table, the norm of a post-norm layer, a norm over spans of columns
# (csrc/elementwise.cu); gated linear attention (csrc/gla.cu)


def embed_pair(tokens: torch.Tensor, positions: torch.Tensor, table: torch.Tensor, pair: torch.Tensor, out: torch.Tensor, *,
               seg_q0: torch.Tensor, seg_qn: torch.Tensor, state_slots: torch.Tensor, last: torch.Tensor, n_seg: int,
               longest_new: int, mul_prev: int, mul_cur: int) -> None:
    """out[t] = table[tok_t] + pair[r_t] as float32, r_t = (prev_t * mul_prev + tok_t * mul_cur) mod buckets with
    buckets = rows of ``pair`` - 1, and r_t = buckets for a token at position 0.  The token before a segment's first one
    is read from ``last`` [n_slots, 1] int32 at the request's state slot; afterwards every segment's last token is
    written there (a second launch)."""
    _i32(tokens, "tokens")
    _i32(positions, "positions")
    _cuda_c(table, "table")
    _cuda_c(pair, "pair")
    _cuda_c(out, "out")
    H = table.shape[1]
    _need(out.dtype == torch.float32 and out.shape[1] == H and pair.shape[1] == H and pair.dtype == table.dtype
          and pair.shape[0] >= 2, "embed_pair: tables and out")
    _need(last.is_cuda and last.dtype == torch.int32 and last.dim() == 2 and last.stride(1) == 1, "embed_pair: last [n_slots, 1] int32")
    code = _lib("elementwise").locus_embed_pair(
        _p(tokens), _p(positions), _p(table), _p(pair), I(dtype_code(table.dtype)), _p(out), _p(seg_q0), _p(seg_qn),
        _p(state_slots), _p(last), LL(last.stride(0)), I(n_seg), I(longest_new), I(H), LL(pair.shape[0] - 1), LL(mul_prev),
        LL(mul_cur), _stream())
    if code == 0:
        _count_launches(1)   # the launch that moves the slots on
    _check(code, "embed_pair")


def layernorm_post(x: torch.Tensor, y: torch.Tensor, alpha: float, w: torch.Tensor, b: torch.Tensor, eps: float,
                   cast: Optional[torch.Tensor] = None) -> None:
    """x <- layer_norm(alpha * x + y) * w + b in place on float32 rows (mean and variance in float32); ``cast``: the new
    rows once more in that buffer's element type."""
    _f32c(x, "layernorm_post: x")
    _f32c(y, "layernorm_post: y")
    _cuda_c(w, "w")
    _cuda_c(b, "b")
    n, H = x.shape
    _need(x.is_contiguous() and y.is_contiguous() and y.shape[0] >= n and y.shape[1] == H and w.numel() == H
          and b.numel() == H and w.dtype == b.dtype, "layernorm_post: shapes")
    if cast is not None:
        _cuda_c(cast, "cast")
        _need(cast.shape[0] >= n and cast.shape[1] == H, "layernorm_post: cast")
    code = _lib("elementwise").locus_layernorm_post(
        _p(x), _p(y), F(alpha), _p(w), _p(b), I(dtype_code(w.dtype)), F(eps), _p(cast),
        I(dtype_code(cast.dtype) if cast is not None else 0), I(n), I(H), _stream())
    _check(code, "layernorm_post")


def span_rmsnorm(x: torch.Tensor, spans, eps: float) -> None:
    """RMS norm in place over spans of columns of the float32 rows ``x``: ``spans`` = one or two (offset, width, weight
    [width]); each span is divided by its own root mean square and multiplied by its weight."""
    _f32c(x, "span_rmsnorm: x")
    _need(1 <= len(spans) <= 2 and x.stride(1) == 1, "span_rmsnorm: one or two spans")
    (o0, n0, w0), (o1, n1, w1) = spans[0], (spans[1] if len(spans) > 1 else (0, 0, None))
    for w, n in ((w0, n0), (w1, n1)):
        if w is not None:
            _cuda_c(w, "w")
            _need(w.numel() == n and w.dtype == w0.dtype, "span_rmsnorm: weights")
    code = _lib("elementwise").locus_span_rmsnorm(_p(x), I(x.stride(0)), I(x.shape[0]), I(o0), I(n0), _p(w0), I(o1), I(n1),
                                                  _p(w1), I(dtype_code(w0.dtype)), F(eps), _stream())
    _check(code, "span_rmsnorm")


GLA_MAX_DIM = 256


def gla_decay(z: torch.Tensor, off: int, n: int, tau: float) -> None:
    """z[:, off : off + n] <- 1 - sigmoid(z)^(1 / tau) in place on float32 rows, as -expm1(-softplus(-z) / tau): what a
    row of the state loses per token (the form :func:`gla_scan` takes: near 1 a decay itself is too coarse in float32)."""
    _f32c(z, "gla_decay: z")
    _need(z.stride(1) == 1 and 0 <= off and off + n <= z.shape[1], "gla_decay: columns")
    code = _lib("gla").locus_gla_decay(_p(z), I(z.stride(0)), I(off), I(n), I(z.shape[0]), F(tau), _stream())
    _check(code, "gla_decay")


def gla_scan(q: torch.Tensor, off_q: int, k: torch.Tensor, off_k: int, v: torch.Tensor, off_v: int, decay: torch.Tensor,
             off_a: int, state: torch.Tensor, state_offset: int, state_slots: torch.Tensor, seg_q0: torch.Tensor,
             seg_qn: torch.Tensor, n_seg: int, out: torch.Tensor, *, n_heads: int, dim: int, v_dim: int, q_scale: float) -> None:
    """Gated linear attention per request and head over every segment's new tokens in order, from and into the request's
    state slot: S <- diag(a_t) S + k_t v_t^T; o_t = S^T q_t * q_scale.  ``q``, ``k``, ``decay`` (1 - a_t, one number per
    key channel: :func:`gla_decay`) and ``v``: float32 row matrices in which head h's columns start at ``off_*`` + h * dim (``off_v`` + h * v_dim);
    head h's state [dim, v_dim] starts ``state_offset`` + h * dim * v_dim floats into a slot of ``state`` [n_slots,
    floats]; ``out`` [T, n_heads * v_dim] float32."""
    for t, name in ((q, "q"), (k, "k"), (v, "v"), (decay, "decay"), (out, "out")):
        _f32c(t, f"gla_scan: {name}")
    _i32(state_slots, "state_slots")
    _need(state.is_cuda and state.dtype == torch.float32 and state.dim() == 2 and state.stride(1) == 1
          and state_offset + n_heads * dim * v_dim <= state.shape[1], "gla_scan: the state does not hold the heads")
    _need(out.shape[1] == n_heads * v_dim and dim <= GLA_MAX_DIM, "gla_scan: out [T, n_heads * v_dim], dim <= 256")
    code = _lib("gla").locus_gla_scan(
        _p(q), I(q.stride(0)), I(off_q), _p(k), I(k.stride(0)), I(off_k), _p(v), I(v.stride(0)), I(off_v), _p(decay),
        I(decay.stride(0)), I(off_a), ctypes.c_void_p(state.data_ptr() + 4 * state_offset), LL(state.stride(0)),
        _p(state_slots), _p(seg_q0), _p(seg_qn), I(n_seg), _p(out), I(out.stride(0)), I(n_heads), I(dim), I(v_dim),
        F(q_scale), _stream())
    _check(code, "gla_scan", f"(heads {n_heads}, dim {dim}, v_dim {v_dim})")


def apply_penalties(logits: torch.Tensor, history: torch.Tensor, repeat: torch.Tensor,
                    freq: torch.Tensor, presence: torch.Tensor) -> None:
    """In place: repetition / frequency / presence penalties over ``history`` [R, n] (-1 = none)."""
    _cuda_c(logits, "logits")
    _i32(history, "history")
    R, V = logits.shape
    _need(logits.dtype == torch.float32, "apply_penalties: float32 logits")
    _need(history.shape[0] == R, "apply_penalties: history rows")
    code = _lib("sampling").locus_apply_penalties(
        _p(logits), LL(logits.stride(0)), I(R), I(V), _p(history), I(history.shape[1]), _p(repeat),
        _p(freq), _p(presence), _stream()
    )
    _check(code, "apply_penalties")


def sample_use_cluster(on: bool) -> None:
    """Let rows of 8,192 to 163,840 tokens be sampled by a cluster of eight blocks per row (the default), or keep
    every row on the one-block kernel.  Both give the same tokens; for tests and measurements."""
    _lib("sampling").locus_sample_use_cluster(I(1 if on else 0))


def sample(logits: torch.Tensor, *, temperature: torch.Tensor, top_k: torch.Tensor,
           top_p: torch.Tensor, min_p: torch.Tensor, seeds: torch.Tensor, counters: torch.Tensor,
           out: torch.Tensor, kept_count: Optional[torch.Tensor] = None) -> None:
    """One token per row of ``logits`` [R, V] float32 (temperature <= 0: arg-max)."""
    _need(logits.is_cuda and logits.dtype == torch.float32 and logits.stride(1) == 1,
          "sample: logits must be float32 CUDA rows")
    R, V = logits.shape
    _i32(out, "out")
    _i32(top_k, "top_k")
    for t, n in ((temperature, "temperature"), (top_p, "top_p"), (min_p, "min_p")):
        _need(t.dtype == torch.float32 and t.numel() >= R and t.is_cuda, f"sample: {n} must be float32 [R]")
    for t, n in ((seeds, "seeds"), (counters, "counters")):
        _need(t.dtype == torch.int64 and t.numel() >= R and t.is_cuda, f"sample: {n} must be int64 [R]")
    code = _lib("sampling").locus_sample(
        _p(logits), LL(logits.stride(0)), I(R), I(V), _p(temperature), _p(top_k), _p(top_p), _p(min_p),
        _p(seeds), _p(counters), _p(out), _p(kept_count), _stream()
    )
    _check(code, "sample")


def modules_for(dtype: torch.dtype) -> list:
    """Kernel modules that a model of element type ``dtype`` needs."""
    return ["elementwise", "gemm_simt", "gemv", "gemm_skinny", "gemm_tc", "attention", "attention_mma", "moe_route", "sampling"]
