"""Python faces of the CUDA kernels.

Every function here checks what it is given (device, dtype, contiguity, sizes),
passes raw pointers and the current stream to the `extern "C"` function of the
same purpose, and raises `KernelError` with the kernel's own message when that
refuses.  Nothing here computes: if the compiled library is missing and cannot be
built, loading it raises `ExtensionMissingError`.
"""
from __future__ import annotations

import ctypes
import os
import re
from dataclasses import dataclass
from typing import List, Optional

import torch

from .csrc import build
from .errors import KernelError

F32, BF16 = 0, 1
PAGE_TOKENS = 64
EPI_NONE, EPI_SOFTCAP, EPI_GATED, EPI_BIAS = 0, 1, 2, 3
ACT_GELU_TANH, ACT_SILU, ACT_CLAMPED_SWISH = 0, 1, 2
ACTIVATIONS = {"gelu_tanh": ACT_GELU_TANH, "silu": ACT_SILU}
BIAS_ACTIVATIONS = {"none": 0, "gelu_erf": 1, "gelu_tanh": 2}      # what EPI_BIAS applies after the bias (or without one)
EXPERT_ACTIVATIONS = {"gated_swish": 0, "relu_square": 1}          # the routed experts' (csrc/moe.cu)
# the clamped form as the products' gated epilogues know it: g logistic(SWISH_ALPHA g) (u + SWISH_SHIFT), the limit a parameter
SWISH_ALPHA, SWISH_SHIFT = 1.702, 1.0
ROPE_STYLES = {"rotate_half": 0, "interleaved": 1}

_p, _i, _f, _l = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong

_CT = {"p": _p, "i": _i, "f": _f, "l": _l}
_EXPORT = re.compile(r'extern\s+"C"\s+int\s+(\w+)\s*\(([^)]*)\)', re.S)


def _parse_signatures(sources) -> dict:
    """Argument types of every `extern "C" int f(...)` in the given .cu files, read
    from the sources themselves so that the Python side cannot drift from them."""
    sigs = {}
    for src in sources:
        with open(os.path.join(build.HERE, src)) as fh:
            text = fh.read()
        for name, args in _EXPORT.findall(text):
            sig = ""
            for a in args.split(","):
                a = a.strip()
                if not a:
                    continue
                if "*" in a or "cudaStream_t" in a:
                    sig += "p"
                elif "long long" in a:
                    sig += "l"
                elif a.startswith("float") or a.startswith("const float"):
                    sig += "f"
                else:
                    sig += "i"
            sigs[name] = sig
    return sigs


def dtype_code(dt: torch.dtype) -> int:
    if dt == torch.float32:
        return F32
    if dt == torch.bfloat16:
        return BF16
    raise KernelError(f"no kernel takes dtype {dt}")


def _ptr(t: Optional[torch.Tensor]):
    return None if t is None else ctypes.c_void_p(t.data_ptr())


_raw_stream = getattr(torch._C, "_cuda_getCurrentRawStream", None)
_device_index: Optional[int] = None


def _stream():
    """The current CUDA stream as a raw handle.  Asked for at every launch, so it goes the
    short way: one call into torch's C layer instead of building a Stream object."""
    global _device_index
    if _raw_stream is None:
        return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)
    if _device_index is None:
        _device_index = torch.cuda.current_device()
    return ctypes.c_void_p(_raw_stream(_device_index))


class Library:
    """A loaded CUDA library with typed entry points."""

    def __init__(self, name: str):
        self.name = name
        self.lib = build.load(name)
        self._signatures = _parse_signatures(build.library_spec(name)[0])
        self._fns = {}
        self._last_error = None
        if hasattr(self.lib, "hos_last_error"):
            self._last_error = self.lib.hos_last_error
            self._last_error.restype = ctypes.c_char_p
            self._last_error.argtypes = []
        # kernels whose bounded waits run out say so in one word of pinned host memory (check_errors)
        for setter in _ERROR_WORD_SETTERS:
            f = getattr(self.lib, setter, None)
            if f is not None and torch.cuda.is_available():
                f.restype, f.argtypes = ctypes.c_int, [ctypes.c_void_p]
                f(ctypes.c_void_p(_error_word().data_ptr()))
        self._set_pdl = getattr(self.lib, "hos_set_pdl", None)
        if self._set_pdl is not None:
            self._set_pdl.restype, self._set_pdl.argtypes = None, [ctypes.c_int]
            self._set_pdl(1 if _launch_ahead else 0)
        _libraries.append(self)

    def fn(self, name: str, signature: Optional[str] = None):
        f = self._fns.get(name)
        if f is None:
            try:
                f = getattr(self.lib, name)
            except AttributeError as e:
                raise KernelError(f"library {self.name} has no function {name}") from e
            sig = signature or self._signatures[name]
            f.argtypes = [_CT[c] for c in sig]
            f.restype = ctypes.c_int
            self._fns[name] = f
        return f

    def call(self, name: str, *args, signature: Optional[str] = None, label: Optional[str] = None) -> None:
        """`label`: what the measurement aid below calls it (a function that runs several kinds of work)."""
        global launch_count
        launch_count += 1
        if _call_times is not None:
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            rc = self.fn(name, signature)(*args)
            e1.record()
            _call_times.append((label or name, e0, e1))
        else:
            rc = self.fn(name, signature)(*args)
        if rc != 0:
            msg = self._last_error() if self._last_error else b""
            raise KernelError((msg or b"").decode(errors="replace") or f"{name} failed with code {rc}")


_libraries: List["Library"] = []
_call_times: Optional[list] = None


def time_calls(on: bool) -> None:
    """Measurement aid: while on, every call into a CUDA library is bracketed by two events on the launching
    stream (not inside a graph capture); `call_times()` adds them up by function."""
    global _call_times
    _call_times = [] if on else None


def call_times() -> dict:
    """{function: (calls, milliseconds in all)} of the calls made since time_calls(True); waits for them."""
    torch.cuda.synchronize()
    out = {}
    for name, e0, e1 in _call_times or []:
        n, ms = out.get(name, (0, 0.0))
        out[name] = (n + 1, ms + e0.elapsed_time(e1))
    if _call_times is not None:
        _call_times.clear()
    return out
_launch_ahead = False

_ERROR_WORD_SETTERS = ("hos_gemm_tc_set_error_word", "hos_attn_decode_set_error_word",
                       "hos_attn_prefill_tc_set_error_word")
GIVE_UP_CODES = {1: "the tcgen05 matrix product", 2: "the decode attention", 3: "the tcgen05 prompt attention"}
_error_word_tensor: Optional[torch.Tensor] = None
_after_give_up = []        # callables that put shared scratch state right after a kernel gave up


def _error_word() -> torch.Tensor:
    """One int32 in pinned host memory (the same address on the device): 0, or the code of the
    kernel whose bounded wait ran out last."""
    global _error_word_tensor
    if _error_word_tensor is None:
        _error_word_tensor = torch.zeros(1, dtype=torch.int32).pin_memory()
    return _error_word_tensor


def on_give_up(fn) -> None:
    """Register what has to be put right when a kernel gave up (counters it left behind)."""
    _after_give_up.append(fn)


def check_errors() -> None:
    """Call after a synchronisation, before a step's result is used: raises KernelError if a kernel of
    the steps that are complete by now gave up a bounded wait (its results are then not to be trusted).
    Costs a read of host memory."""
    w = _error_word_tensor
    if w is None:
        return
    code = int(w[0])
    if code == 0:
        return
    w[0] = 0
    for fn in _after_give_up:
        fn()
    raise KernelError(f"{GIVE_UP_CODES.get(code, 'a kernel')} gave up a wait that should have ended (about a second); "
                      f"the results of the steps since the last check are not valid")


_room_left = False


def note_room_left(left: bool) -> None:
    """A launcher's word about the kernel it has just launched: it leaves at least half of the SMs free (the decode
    attention of one sequence does: 64 CTAs).  The launcher of the next kernel may then place that kernel beside it,
    ahead of its end (`take_room_left`); with the SMs full, kernels that wait on them cost more than they hide."""
    global _room_left
    _room_left = bool(left)


def take_room_left() -> bool:
    """What the last launcher said (see note_room_left); the word holds for one launch."""
    global _room_left
    left, _room_left = _room_left, False
    return left


def set_launch_ahead(on: bool) -> None:
    """Whether kernels are launched so that they may be set up while the kernel before them still
    runs (programmatic dependent launch).  It pays for steps of many tokens, whose kernels are
    launched one by one, and costs for single-token steps; the runner switches it per step."""
    global _launch_ahead
    if on == _launch_ahead:
        return
    _launch_ahead = on
    for lib in _libraries:
        if lib._set_pdl is not None:
            lib._set_pdl(1 if on else 0)


_sm_count: Optional[int] = None


def sm_count() -> int:
    """Streaming multiprocessors of the current device (asked once).  Without a device, as the
    host-side choices are also exercised where there is none, the B200's 148."""
    global _sm_count
    if _sm_count is None:
        _sm_count = (torch.cuda.get_device_properties(torch.cuda.current_device()).multi_processor_count
                     if torch.cuda.is_available() else 148)
    return _sm_count


_core: Optional[Library] = None
launch_count = 0        # calls into the CUDA libraries so far (each launches one kernel or more)


def core() -> Library:
    global _core
    if _core is None:
        _core = Library("core")
    return _core


def _check(t: torch.Tensor, what: str, dtype=None, dim=None) -> None:
    if not t.is_cuda:
        raise KernelError(f"{what} must be on the GPU")
    if dtype is not None and t.dtype != dtype:
        raise KernelError(f"{what} must be {dtype}, found {t.dtype}")
    if dim is not None and t.dim() != dim:
        raise KernelError(f"{what} must have {dim} dimensions, found {t.dim()}")
    if not t.is_contiguous():
        raise KernelError(f"{what} must be contiguous")


@dataclass
class PagedKVArgs:
    """One call's view of the paged cache, as the kernels take it."""
    k_pages: torch.Tensor        # [n_pages, n_kv_heads, 64, head_dim]
    v_pages: torch.Tensor
    page_table: torch.Tensor     # int32 [n_slots, table_stride]
    ring_pages: int              # 0: all keys kept; > 0: ring of that many pages
    n_kv_heads: int
    head_dim: int
    v_head_dim: int = 0          # 0: values are as wide as keys

    @property
    def table_stride(self) -> int:
        return self.page_table.shape[1]

    @property
    def v_dim(self) -> int:
        return self.v_head_dim or self.head_dim


# ---- element-wise and norms ------------------------------------------------------------

def embed(tokens: torch.Tensor, table: torch.Tensor, scale: float, out: torch.Tensor, copies: int = 1) -> None:
    """out[n] = `copies` copies of table[token] * scale, side by side."""
    _check(tokens, "tokens", torch.int32, 1)
    _check(table, "embedding table", None, 2)
    _check(out, "embedding output", torch.float32, 2)
    n, d = out.shape[0], table.shape[1]
    if tokens.shape[0] != n or out.shape[1] != copies * d:
        raise KernelError("embed: sizes of tokens, table and output disagree")
    core().call("hos_embed", _ptr(tokens), _ptr(table), dtype_code(table.dtype), float(scale),
                _ptr(out), n, d, int(copies), _stream())


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, add_one: bool, out: torch.Tensor) -> None:
    _check(x, "norm input", None, 2)
    _check(w, "norm weight", torch.float32, 1)
    _check(out, "norm output", None, 2)
    n, d = x.shape
    if out.shape != x.shape or w.shape[0] != d:
        raise KernelError("rmsnorm: sizes of input, weight and output disagree")
    core().call("hos_rmsnorm", _ptr(x), dtype_code(x.dtype), _ptr(w), float(eps), int(add_one),
                _ptr(out), dtype_code(out.dtype), n, d, _stream())


def norm_add_norm(y: torch.Tensor, w_post: torch.Tensor, eps_post: float, add_one_post: bool,
                  x: torch.Tensor, w_next: Optional[torch.Tensor] = None, eps_next: float = 0.0,
                  add_one_next: bool = False, h: Optional[torch.Tensor] = None) -> None:
    """x += RMSNorm(y; w_post); if h is given, h = RMSNorm(x; w_next), or x itself in h's type without w_next.  y is [N, D], or
    [parts, N, D] float32 partial sums (of a matrix product that split K), added here."""
    _check(y, "norm input")
    _check(x, "residual stream", torch.float32, 2)
    _check(w_post, "norm weight", torch.float32, 1)
    n_parts = y.shape[0] if y.dim() == 3 else 1
    n, d = x.shape
    if tuple(y.shape[-2:]) != (n, d) or w_post.shape[0] != d or y.dim() not in (2, 3):
        raise KernelError("norm_add_norm: sizes disagree")
    if h is not None:
        _check(h, "next norm output", None, 2)
        if w_next is not None:
            _check(w_next, "next norm weight", torch.float32, 1)
        if h.shape != x.shape or (w_next is not None and w_next.shape[0] != d):
            raise KernelError("norm_add_norm: sizes of the next norm disagree")
    core().call("hos_norm_add_norm", _ptr(y), dtype_code(y.dtype), n_parts, _ptr(w_post), float(eps_post),
                int(add_one_post), _ptr(x), _ptr(w_next), float(eps_next), int(add_one_next),
                _ptr(h), dtype_code(h.dtype) if h is not None else 0, n, d, _stream())


def rope_table(token_pos: torch.Tensor, inv_freq: torch.Tensor) -> torch.Tensor:
    """float32 [N, len(inv_freq), 2]: (cos, sin) of position * inv_freq, taken in 32-bit."""
    _check(token_pos, "positions", torch.int32, 1)
    _check(inv_freq, "inverse frequencies", torch.float32, 1)
    out = torch.empty((token_pos.shape[0], inv_freq.shape[0], 2), dtype=torch.float32, device=token_pos.device)
    core().call("hos_rope_table", _ptr(token_pos), _ptr(inv_freq), _ptr(out), token_pos.shape[0], inv_freq.shape[0],
                _stream())
    return out


def residual_add(y: torch.Tensor, x: torch.Tensor) -> None:
    _check(y, "branch output")
    _check(x, "residual stream", torch.float32)
    if y.shape != x.shape:
        raise KernelError("residual_add: sizes disagree")
    core().call("hos_residual_add", _ptr(y), dtype_code(y.dtype), _ptr(x), x.numel(), _stream())


def rope_kv_write(qkv: torch.Tensor, n_heads: int, token_pos, token_seq, seq_slot, seq_len_after,
                  inv_freq: Optional[torch.Tensor], rotary_dim: int, style: int,
                  cache: Optional[PagedKVArgs], n_kv_heads: int, head_dim: int,
                  partials: Optional[torch.Tensor] = None) -> None:
    """Rotate the q and k heads of the fused projection rows `qkv` in place; if `cache` is
    given, store the rotated keys and the values at the tokens' places.  With `partials`
    ([parts, N, width] float32 partial sums of the projection) the rows are first formed from
    them and written to `qkv`."""
    _check(qkv, "qkv rows", None, 2)
    n, stride = qkv.shape
    if stride != (n_heads + 2 * n_kv_heads) * head_dim:
        raise KernelError("rope: row width does not match the head counts")
    if inv_freq is None:
        rotary_dim = 0
    else:
        _check(inv_freq, "inverse frequencies", torch.float32, 1)
        if inv_freq.shape[0] * 2 != rotary_dim:
            raise KernelError("rope: one inverse frequency per rotated pair is needed")
    if cache is not None and cache.k_pages.dtype != qkv.dtype:
        raise KernelError("rope: cache and activations differ in dtype")
    src, n_parts = qkv, 1
    if partials is not None:
        _check(partials, "partial sums", torch.float32, 3)
        if tuple(partials.shape[1:]) != (n, stride):
            raise KernelError("rope: partial sums and rows differ in size")
        src, n_parts = partials, partials.shape[0]
    core().call("hos_rope_kv_write", _ptr(src), dtype_code(src.dtype), n_parts, _ptr(qkv), dtype_code(qkv.dtype),
                stride, n_heads,
                _ptr(token_pos), _ptr(token_seq), _ptr(seq_slot), _ptr(seq_len_after),
                _ptr(inv_freq), rotary_dim, style,
                _ptr(cache.k_pages) if cache else None, _ptr(cache.v_pages) if cache else None,
                _ptr(cache.page_table) if cache else None, cache.table_stride if cache else 0,
                cache.ring_pages if cache else 0, n_kv_heads, head_dim, 1 if cache else 0, n,
                _stream())


def gated_act(gu: torch.Tensor, out: torch.Tensor, act: int) -> None:
    _check(gu, "gate|up rows", None, 2)
    _check(out, "activation output", gu.dtype, 2)
    n, f = out.shape
    if gu.shape != (n, 2 * f):
        raise KernelError("gated_act: sizes disagree")
    core().call("hos_gated_act", _ptr(gu), _ptr(out), dtype_code(gu.dtype), n, f, act, _stream())


def clamped_gated_act(gu: torch.Tensor, out: torch.Tensor, limit: float, alpha: float, shift: float) -> None:
    """out = g logistic(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, -limit, limit) (limit 0: no clamp);
    gu: float32 [N, 2F] gate then up; out: [N, F] in the products' type."""
    _check(gu, "gate|up rows", torch.float32, 2)
    n, f = out.shape
    if gu.shape != (n, 2 * f):
        raise KernelError("clamped_gated_act: sizes disagree")
    core().call("hos_clamped_gated_act", _ptr(gu), _ptr(out), dtype_code(out.dtype), n, f, float(limit), float(alpha),
                float(shift), _stream())


def gather_rows(x: torch.Tensor, idx: torch.Tensor, out: torch.Tensor) -> None:
    _check(x, "rows", torch.float32, 2)
    _check(idx, "row indices", torch.int32, 1)
    _check(out, "gathered rows", torch.float32, 2)
    if out.shape != (idx.shape[0], x.shape[1]):
        raise KernelError("gather_rows: sizes disagree")
    core().call("hos_gather_rows", _ptr(x), _ptr(idx), _ptr(out), idx.shape[0], x.shape[1], _stream())


# ---- matrix product (plain) --------------------------------------------------------------

def gemm_plain(a: torch.Tensor, w: torch.Tensor, out: torch.Tensor, epilogue: int = EPI_NONE,
               cap: float = 0.0, act: int = 0, bias: Optional[torch.Tensor] = None) -> None:
    """out[M, N] = a[M, K] . w[N, K]^T with 32-bit accumulation on the CUDA cores.
    Gated epilogue: w has 2N rows (gate rows, then up rows), out = act(gate) * up.  Bias epilogue: act(product + bias),
    or act(product) with no bias."""
    _check(a, "left operand", None, 2)
    _check(w, "weight", None, 2)
    _check(out, "product", None, 2)
    m, k = a.shape
    n = out.shape[1]
    want_rows = 2 * n if epilogue == EPI_GATED else n
    if out.shape[0] != m or w.shape != (want_rows, k):
        raise KernelError(f"gemm: sizes disagree: a {tuple(a.shape)} w {tuple(w.shape)} out {tuple(out.shape)}")
    core().call("hos_gemm_plain", _ptr(a), dtype_code(a.dtype), _ptr(w), dtype_code(w.dtype),
                _ptr(out), dtype_code(out.dtype), m, n, k, k, k, n, epilogue, float(cap), act, _ptr(bias),
                _stream())


# ---- attention (plain) -------------------------------------------------------------------

def attn_plain(q: torch.Tensor, q_stride: int, out: torch.Tensor, token_pos, token_seq, n_tokens: int,
               n_heads: int, n_kv_heads: int, head_dim: int, scale: float, cap: float,
               window: Optional[int], *, k_rows=None, v_rows=None, kv_stride: int = 0,
               cu_seqlens=None, seq_slot=None, cache: Optional[PagedKVArgs] = None) -> None:
    """Either (k_rows, v_rows, cu_seqlens): keys of this step's own rows, sequences
    from position 0; or (cache, seq_slot): keys from the paged cache."""
    paged = cache is not None
    _check(out, "attention output", q.dtype, 2)
    core().call("hos_attn_plain", dtype_code(q.dtype), int(paged), _ptr(q), q_stride,
                _ptr(k_rows), _ptr(v_rows), kv_stride, _ptr(out), out.shape[1],
                _ptr(token_pos), _ptr(token_seq), _ptr(cu_seqlens), _ptr(seq_slot),
                _ptr(cache.k_pages) if paged else None, _ptr(cache.v_pages) if paged else None,
                _ptr(cache.page_table) if paged else None, cache.table_stride if paged else 0,
                cache.ring_pages if paged else 0, n_tokens, n_heads, n_kv_heads, head_dim,
                float(scale), float(cap), int(window) if window else 0, _stream())


# ---- sampling ----------------------------------------------------------------------------

_argmax_state = {}


def argmax(logits: torch.Tensor, out: torch.Tensor, rep_penalty: float = 1.0,
           recent: Optional[torch.Tensor] = None, recent_len: Optional[torch.Tensor] = None) -> None:
    """out[b] = the first maximum of row b.  With `recent` ([B, n] token ids, recent_len[b] of them
    valid) and a penalty other than 1 the sampler's repetition penalty is applied on the fly."""
    _check(logits, "logits", torch.float32, 2)
    _check(out, "tokens", torch.int32, 1)
    b, v = logits.shape
    stride = 0
    if recent is not None:
        _check(recent, "recent tokens", torch.int32, 2)
        _check(recent_len, "recent counts", torch.int32, 1)
        if recent.shape[0] != b or recent_len.shape[0] != b:
            raise KernelError("argmax: one row of recent tokens per row of logits is needed")
        stride = recent.shape[1]
    lib = core()
    f = lib.lib.hos_argmax_chunks
    f.restype, f.argtypes = ctypes.c_int, [ctypes.c_int]
    chunks = f(v)
    key = (logits.device, b, chunks)
    st = _argmax_state.get(key)
    if st is None:       # partial maxima and ids, and the tickets (zero between launches)
        st = _argmax_state[key] = (torch.empty(2 * b * chunks, dtype=torch.float32, device=logits.device),
                                   torch.zeros(b, dtype=torch.int32, device=logits.device))
    lib.call("hos_argmax", _ptr(logits), v, b, v, _ptr(out), _ptr(st[0]), _ptr(st[1]), _ptr(recent), stride,
             _ptr(recent_len), float(rep_penalty), _stream())


def sample(logits: torch.Tensor, uniforms: torch.Tensor, out: torch.Tensor, temp: float, top_k: int,
           top_p: float, rep_penalty: float = 1.0, recent: Optional[torch.Tensor] = None,
           recent_len: Optional[torch.Tensor] = None) -> None:
    _check(logits, "logits", torch.float32, 2)
    _check(uniforms, "uniform draws", torch.float32, 1)
    _check(out, "tokens", torch.int32, 1)
    b, v = logits.shape
    if recent is not None:
        _check(recent, "recent tokens", torch.int32, 2)
        _check(recent_len, "recent lengths", torch.int32, 1)
    core().call("hos_sample", _ptr(logits), v, b, v, _ptr(uniforms), _ptr(recent),
                recent.shape[1] if recent is not None else 0, _ptr(recent_len), float(temp),
                int(top_k), float(top_p), float(rep_penalty), _ptr(out), _stream())


# ---- the per-slot record (csrc/slot_state.cu) ----------------------------------------------
SLOT_WORDS, RECENT_MAX, MAX_STOPS = 8, 256, 16
SLOT_POS, SLOT_LAST, SLOT_FLAGS, SLOT_COUNT, SLOT_RNG_LO, SLOT_RNG_HI, SLOT_LIMIT = range(7)
BEGIN_ADVANCE, BEGIN_TOKEN_FROM_RECORD, BEGIN_UNIFORM, BEGIN_RECENT, BEGIN_SKIP_FINISHED = 1, 2, 4, 8, 16


def slot_begin(record, ring, slots, meta, b: int, flags: int, tokens, pos, after, seq, cu, uniforms=None,
               recent=None, recent_len=None) -> None:
    """The start of a single-token step of up to b rows (meta[0] of them live): row i belongs to slot
    slots[i]; positions come from the record and move on by one; the input token comes from the
    record (or stays the caller's); for sampling, the next draw of each sequence's generator and its
    recent tokens."""
    core().call("hos_slot_begin", _ptr(record), _ptr(ring), _ptr(slots), _ptr(meta), int(b), int(flags), _ptr(tokens),
                _ptr(pos), _ptr(after), _ptr(seq), _ptr(cu), _ptr(uniforms), _ptr(recent), _ptr(recent_len),
                recent.shape[1] if recent is not None else 0, _stream())


def slot_end(record, ring, slots, meta, b: int, sampled) -> None:
    """After sampling: the tokens go into the records (last token, recent tokens, count, finished)."""
    core().call("hos_slot_end", _ptr(record), _ptr(ring), _ptr(slots), _ptr(meta), int(b), _ptr(sampled), _stream())


def slot_set_pos(record, seq_slot, seq_len_after, cu_seqlens, n_seqs: int) -> None:
    core().call("hos_slot_set_pos", _ptr(record), _ptr(seq_slot), _ptr(seq_len_after), _ptr(cu_seqlens), int(n_seqs),
                _stream())


def slot_write(record, slots, values, word_mask: int) -> None:
    """record[slots[i]][w] = values[i][w] for the words w whose bit is set in word_mask."""
    _check(values, "record values", torch.int32, 2)
    core().call("hos_slot_write", _ptr(record), _ptr(slots), _ptr(values), int(word_mask), values.shape[0], _stream())


def decode_advance(tokens, token_pos, seq_len_after, token_seq, sampled) -> None:
    core().call("hos_decode_advance", _ptr(tokens), _ptr(token_pos), _ptr(seq_len_after), _ptr(token_seq),
                _ptr(sampled), tokens.shape[0], _stream())


# ---- the other kinds of block (csrc/embed_pair.cu, latent_attention.cu, wkv.cu, moe.cu) ------
_blocks: Optional[Library] = None


def blocks() -> Library:
    """Attention over a latent cache and the matrix-state recurrence with its token shift."""
    global _blocks
    if _blocks is None:
        _blocks = Library("blocks")
    return _blocks


_rows_lib: Optional[Library] = None
_experts: Optional[Library] = None
_gated_attn_lib: Optional[Library] = None


def rows_lib() -> Library:
    """The hashed token-pair embedding, the parallel block's add-and-norms, the norm without statistics."""
    global _rows_lib
    if _rows_lib is None:
        _rows_lib = Library("rows")
    return _rows_lib


def experts() -> Library:
    """The routed feed-forward."""
    global _experts
    if _experts is None:
        _experts = Library("experts")
    return _experts


def gated_attn_lib() -> Library:
    """Attention with a gate per head, a sink, chunks or a window, keys and values of unequal sizes."""
    global _gated_attn_lib
    if _gated_attn_lib is None:
        _gated_attn_lib = Library("gated_attn")
    return _gated_attn_lib


def embed_pair(step, prev_token: torch.Tensor, table: torch.Tensor, pair_table: torch.Tensor, buckets: int,
               mul_prev: int, mul_cur: int, out: torch.Tensor) -> None:
    """out[n] = table[token] + pair_table[(previous * mul_prev + token * mul_cur) % buckets], row `buckets`
    for a sequence's first token; the previous token of a continuing sequence's first row is
    prev_token[slot].  `step`: a StepInfo (device arrays)."""
    _check(out, "embedding output", torch.float32, 2)
    _check(prev_token, "previous tokens", torch.int32, 1)
    n, d = out.shape
    if table.dtype != pair_table.dtype or table.shape[1] != d or pair_table.shape != (buckets + 1, d):
        raise KernelError("embed_pair: the tables do not fit each other or the output")
    rows_lib().call("hos_embed_pair", _ptr(step.tokens), _ptr(step.token_pos), _ptr(step.token_seq),
                  _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(prev_token), _ptr(table), _ptr(pair_table),
                  dtype_code(table.dtype), int(buckets), int(mul_prev), int(mul_cur), _ptr(out), n, d, _stream())


def keep_last_token(step, prev_token: torch.Tensor) -> None:
    rows_lib().call("hos_keep_last_token", _ptr(step.tokens), _ptr(step.token_seq), _ptr(step.cu_seqlens),
                  _ptr(step.seq_slot), _ptr(prev_token), int(step.n_seqs), _stream())


def scaled_add_norms(a: Optional[torch.Tensor], f: Optional[torch.Tensor], mult: float, x: torch.Tensor,
                     w1: Optional[torch.Tensor] = None, eps1: float = 0.0, h1: Optional[torch.Tensor] = None,
                     w2: Optional[torch.Tensor] = None, eps2: float = 0.0, h2: Optional[torch.Tensor] = None) -> None:
    """x += mult * (a + f) (either may be absent); then h1 = RMSNorm(x; w1, eps1), h2 = RMSNorm(x; w2, eps2)
    for those that are given."""
    _check(x, "residual stream", torch.float32, 2)
    n, d = x.shape
    for t, what in ((a, "mixer output"), (f, "feed-forward output"), (h1, "first norm output"), (h2, "second norm output")):
        if t is not None:
            _check(t, what, None, 2)
            if t.shape != x.shape:
                raise KernelError(f"scaled_add_norms: {what} and the residual stream differ in size")
    if h1 is not None and h2 is not None and h1.dtype != h2.dtype:
        raise KernelError("scaled_add_norms: the two norm outputs differ in dtype")
    h = h1 if h1 is not None else h2
    rows_lib().call("hos_scaled_add_norms", _ptr(a), dtype_code(a.dtype) if a is not None else 0,
                  _ptr(f), dtype_code(f.dtype) if f is not None else 0, float(mult), _ptr(x),
                  _ptr(w1), float(eps1), _ptr(h1), _ptr(w2), float(eps2), _ptr(h2),
                  dtype_code(h.dtype) if h is not None else 0, n, d, _stream())


def latent_prep(step, rank: int, rot: int, eps: float, inv_freq: Optional[torch.Tensor], rot_dims: int, style: int, down=None,
                w_norm: Optional[torch.Tensor] = None, kc: Optional[torch.Tensor] = None, cache: Optional[PagedKVArgs] = None,
                cq=None, cq_norm: Optional[torch.Tensor] = None, cq_out: Optional[torch.Tensor] = None) -> None:
    """Norms, the key part's rotation and the cache write between the down projections and what reads their latents.  `down`
    and `cq` are (rows, first column) or None: the latent and the shared key part [rank + rot] -> kc and the cache; the
    queries' own latent -> cq_out, normed with cq_norm.  style: the rotation's pairing (ROPE_STYLES)."""
    rows = next((p[0] for p in (down, cq) if p is not None), None)
    if rows is None:
        raise KernelError("latent_prep: no rows")
    n, dt = rows.shape[0], rows.dtype
    rq = cq_out.shape[1] if cq_out is not None else 0
    for part, cols, what in ((down, rank + rot, "latent rows"), (cq, rq, "query latents")):
        if part is not None:
            _check(part[0], what, dt, 2)
            if part[0].shape[0] != n or part[1] + cols > part[0].shape[1]:
                raise KernelError(f"latent_prep: sizes of the {what} disagree")
    if down is not None:
        _check(kc, "latent rows", dt, 2)
        if kc.shape != (n, rank + rot) or w_norm is None or w_norm.shape[0] != rank:
            raise KernelError("latent_prep: sizes disagree")
    else:
        cache = None
    if cq is not None:
        _check(cq_out, "normed query latents", dt, 2)
        if cq_out.shape[0] != n or cq_norm is None or cq_norm.shape[0] != rq:
            raise KernelError("latent_prep: sizes disagree")
    if cache is not None and (cache.k_pages.dtype != dt or cache.head_dim != rank + rot or cache.n_kv_heads != 1):
        raise KernelError("latent_prep: the cache does not fit the latent rows")

    def at(part):
        if part is None:
            return None, 0
        return ctypes.c_void_p(part[0].data_ptr() + part[1] * part[0].element_size()), part[0].shape[1]
    blocks().call("hos_latent_prep", *at(down), *at(cq), dtype_code(dt), rank, rot, rq, _ptr(w_norm), _ptr(cq_norm), float(eps),
                  _ptr(inv_freq), int(rot_dims) if inv_freq is not None else 0, int(style), _ptr(step.token_pos),
                  _ptr(step.token_seq), _ptr(step.seq_slot), _ptr(step.seq_len_after), _ptr(kc) if down is not None else None,
                  _ptr(cq_out), _ptr(cache.k_pages) if cache else None, _ptr(cache.page_table) if cache else None,
                  cache.table_stride if cache else 0, cache.ring_pages if cache else 0, n, _stream())


def latent_attn(q_lat: torch.Tensor, q: torch.Tensor, dq: int, inv_freq: Optional[torch.Tensor], rot_dims: int, style: int, kc: Optional[torch.Tensor], cache: Optional[PagedKVArgs], sink: Optional[torch.Tensor],
                o_lat: torch.Tensor, step, row0: int, rows: int, rank: int, scale: float, window: Optional[int],
                paged: bool, n_splits: int = 1, rows_per_block: int = 1, tensor_cores: bool = True) -> None:
    """q_lat: float32 [N, heads, rank], the queries' unrotated parts taken to the latent; q: rows whose first columns are the
    heads' queries as projected, dq unrotated and then the rotated numbers each (rotated here; style: ROPE_STYLES).
    Rows row0 .. row0+rows-1 of the step: keys from `kc` (the step's own rows; sequences from position 0)
    or from the paged cache.  `n_splits` > 1: every row's keys are cut into that many shares that run side by side
    and are merged (few rows: decoding); `rows_per_block` > 1: neighbouring rows share the keys they read (prompts)."""
    _check(q_lat, "latent queries", torch.float32, 3)
    _check(o_lat, "latent outputs", (cache.k_pages if paged else kc).dtype, 3)
    n, heads, r = q_lat.shape
    src = cache.k_pages if paged else kc
    _check(q, "query rows", src.dtype, 2)
    d = src.shape[-1]
    if r != rank or o_lat.shape != (n, heads, rank) or q.shape[0] != n or q.shape[1] < heads * (dq + d - rank):
        raise KernelError("latent_attn: sizes disagree")
    part_acc = part_ml = None
    if n_splits > 1:
        part_acc = torch.empty((n, heads, n_splits, rank), dtype=torch.float32, device=q_lat.device)
        part_ml = torch.empty((n, heads, n_splits, 2), dtype=torch.float32, device=q_lat.device)
    blocks().call("hos_latent_attn", dtype_code(src.dtype), int(paged), _ptr(q_lat), _ptr(q), q.shape[1], int(dq), _ptr(inv_freq),
                  int(rot_dims) if inv_freq is not None else 0, int(style), _ptr(kc),
                  _ptr(cache.k_pages) if paged else None, _ptr(cache.page_table) if paged else None,
                  cache.table_stride if paged else 0, cache.ring_pages if paged else 0, _ptr(sink), _ptr(o_lat),
                  _ptr(part_acc), _ptr(part_ml), int(n_splits), int(rows_per_block),
                  _ptr(step.token_pos), _ptr(step.token_seq), _ptr(step.cu_seqlens), _ptr(step.seq_slot),
                  int(row0), int(rows), heads, rank, d, float(scale), int(window) if window else 0,
                  1 if tensor_cores else 0, _stream())


def heads_product(x: torch.Tensor, x_off: int, lda: int, a_head: int, w: torch.Tensor, out: torch.Tensor, out_off: int,
                  ldo: int, o_head: int, m: int) -> None:
    """out[r, h, :] = w[h] . x[r, h, :] for all heads in one launch; w: [heads, N, K]; x and out are given with
    an element offset, a row stride and a head stride (in elements)."""
    heads, n, k = w.shape
    blocks().call("hos_heads_product", ctypes.c_void_p(x.data_ptr() + x_off * x.element_size()), dtype_code(x.dtype),
                  _ptr(w), dtype_code(w.dtype), ctypes.c_void_p(out.data_ptr() + out_off * out.element_size()),
                  dtype_code(out.dtype), int(m), n, k, heads, int(lda), int(a_head), int(ldo), int(o_head), _stream())


def token_shift(h: torch.Tensor, kept: torch.Tensor, mu: torch.Tensor, step) -> List[torch.Tensor]:
    """The mixes h + (previous row - h) * mu[s], one [N, D] tensor per row of mu (each 16-byte aligned)."""
    _check(h, "rows", None, 2)
    _check(mu, "mixing weights", torch.float32, 2)
    n, d = h.shape
    if mu.shape[1] != d or kept.shape[1] != d:
        raise KernelError("token_shift: sizes disagree")
    plane = (n * d + 15) // 16 * 16
    out = torch.empty(mu.shape[0] * plane, dtype=h.dtype, device=h.device)
    blocks().call("hos_token_shift", _ptr(h), dtype_code(h.dtype), _ptr(kept), _ptr(mu), mu.shape[0],
                  _ptr(step.token_pos), _ptr(step.token_seq), _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(out),
                  plane, n, d, _stream())
    return [out[s * plane: s * plane + n * d].view(n, d) for s in range(mu.shape[0])]


def tanh_rows(x: torch.Tensor, out: torch.Tensor) -> None:
    _check(x, "rows", torch.float32)
    _check(out, "tanh output")
    blocks().call("hos_tanh_rows", _ptr(x), _ptr(out), dtype_code(out.dtype), x.numel(), _stream())


def wkv_scan(r, k, v, wx, g, w0, u, norm_w, eps: float, state: torch.Tensor, kept: torch.Tensor, h: torch.Tensor,
             step, out: torch.Tensor, heads: int, dim: int) -> None:
    for t in (r, k, v, wx, g):
        _check(t, "recurrence input", torch.float32, 2)
        if t.shape != (h.shape[0], heads * dim):
            raise KernelError("wkv_scan: sizes disagree")
    _check(state, "recurrent state", torch.float32, 4)
    _check(out, "recurrence output", h.dtype, 2)
    blocks().call("hos_wkv_scan", _ptr(r), _ptr(k), _ptr(v), _ptr(wx), _ptr(g), _ptr(w0), _ptr(u), _ptr(norm_w),
                  float(eps), _ptr(state), _ptr(kept), _ptr(h), dtype_code(h.dtype), h.shape[1], _ptr(step.token_pos),
                  _ptr(step.token_seq), _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(out), int(step.n_seqs),
                  heads, dim, _stream())


_moe_tile: Optional[int] = None


def moe_tile_rows() -> int:
    global _moe_tile
    if _moe_tile is None:
        f = experts().lib.hos_moe_tile_rows
        f.restype, f.argtypes = ctypes.c_int, []
        _moe_tile = int(f())
    return _moe_tile


MOE_SCORING = {"softmax": 0, "logistic": 1}


def moe_route(h, router, correction, token_seq, choice, weight, top: int, scoring: int = 0,
              renormalise: Optional[float] = None, weight_scale: float = 1.0, groups: Optional[tuple] = None) -> None:
    """renormalise (a number >= 0): the chosen scores are divided by their sum plus that number; weight_scale: a constant
    on every weight after that.  groups (count, keep): only outputs of the `keep` best of `count` equal groups can be chosen."""
    _check(h, "rows", None, 2)
    _check(router, "router", torch.float32, 2)
    n, d = h.shape
    # few rows and many router outputs: the outputs are cut over blocks, which leave their logits here for a second launch
    logits = torch.empty((n, router.shape[0]), dtype=torch.float32, device=h.device) if router.shape[0] > 8 and n < 2048 else None
    experts().call("hos_moe_route", _ptr(h), dtype_code(h.dtype), _ptr(router), _ptr(correction), _ptr(token_seq),
                  _ptr(choice), _ptr(weight), n, d, router.shape[0], int(top), int(scoring), _ptr(logits),
                  -1.0 if renormalise is None else float(renormalise), float(weight_scale), *(groups or (0, 0)), _stream())


def moe_align(choice, n_experts: int, listed, tile_expert) -> None:
    experts().call("hos_moe_align", _ptr(choice), choice.numel(), int(n_experts), _ptr(listed), listed.numel(),
                  _ptr(tile_expert), tile_expert.numel(), _stream())


def moe_gate_up(h, w, listed, tile_expert, y, top: int, limit: float, alpha: float, up_shift: float = 1.0,
                in_weight: Optional[torch.Tensor] = None, act: int = 0) -> None:
    """w: [experts, 2F, D], gate rows then up rows, or [experts, F, D] for an activation without a gate (act, one of
    EXPERT_ACTIVATIONS).  in_weight ([pairs] float32): the pair's weight multiplies the expert's input (then `moe_down` takes
    none)."""
    _check(w, "expert gate/up weights", h.dtype, 3)
    if w.shape[1] != y.shape[1] * (2 if act == 0 else 1):
        raise KernelError("moe_gate_up: the experts' weights do not fit the inner rows")
    experts().call("hos_moe_gate_up", _ptr(h), _ptr(w), dtype_code(h.dtype), _ptr(listed), _ptr(tile_expert), _ptr(y),
                  tile_expert.numel(), h.shape[1], y.shape[1], int(top), float(limit), float(alpha), float(up_shift),
                  _ptr(in_weight), int(act), _stream())


def moe_down(y, w, listed, tile_expert, weight, pair_out) -> None:
    _check(w, "expert down weights", y.dtype, 3)
    experts().call("hos_moe_down", _ptr(y), _ptr(w), dtype_code(y.dtype), _ptr(listed), _ptr(tile_expert), _ptr(weight),
                  _ptr(pair_out), tile_expert.numel(), w.shape[1], w.shape[2], _stream())


def moe_few(h, w_gate_up, w_down, choice, weight, y, pair_out, top: int, n_experts: int, limit: float, alpha: float,
            up_shift: float = 1.0, weight_on_input: bool = False, act: int = 0) -> bool:
    """Both expert products for a handful of (row, choice) pairs, without lists or tiles (decoding at small batch):
    y [pairs, F] and pair_out [pairs, D] by pair id.  False: the sizes are not these kernels' and nothing ran."""
    lib = experts()
    global launch_count
    pairs, d, f = choice.numel(), h.shape[1], w_down.shape[2]

    def timed(name, *args):                 # these calls may answer 1 (not their sizes), so they do not go through call()
        if _call_times is None:
            return lib.fn(name)(*args)
        e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        e0.record()
        rc = lib.fn(name)(*args)
        e1.record()
        if rc == 0:
            _call_times.append((name, e0, e1))
        return rc

    rc = timed("hos_moe_gate_up_few", _ptr(h), _ptr(w_gate_up), _ptr(choice), _ptr(y), pairs, d, f, int(top), int(n_experts),
               float(limit), float(alpha), float(up_shift), _ptr(weight) if weight_on_input else None, int(act), _stream())
    if rc == 1:
        return False
    if rc == 0:
        rc = timed("hos_moe_down_few", _ptr(y), _ptr(w_down), _ptr(choice), None if weight_on_input else _ptr(weight),
                   _ptr(pair_out), pairs, d, f, int(n_experts), _stream())
    launch_count += 2
    if rc != 0:
        msg = lib._last_error() if lib._last_error else b""
        raise KernelError((msg or b"").decode(errors="replace") or "the few-rows expert products failed")
    return True


def moe_combine(pair_out, choice, weight, h, out, top: int, n_experts: int, extra: Optional[torch.Tensor] = None) -> None:
    """extra ([N, D] of h's type): added to every row (an expert that all rows use)."""
    n, d = h.shape
    if extra is not None:
        _check(extra, "the shared expert's output", h.dtype, 2)
        if extra.shape != h.shape:
            raise KernelError("moe_combine: the shared expert's output and the rows differ in size")
    experts().call("hos_moe_combine", _ptr(pair_out), _ptr(choice), _ptr(weight), _ptr(h), dtype_code(h.dtype), _ptr(out),
                  n, d, int(top), int(n_experts), _ptr(extra), _stream())


def add_dyt(a: Optional[torch.Tensor], f: Optional[torch.Tensor], mult: float, x: torch.Tensor, alpha: float,
            w: Optional[torch.Tensor], b: Optional[torch.Tensor], h: Optional[torch.Tensor]) -> None:
    """x += mult * (a + f) (either may be absent; each [N, D] of any type or [parts, N, D] float32 partial sums); then,
    if h is given, h = tanh(alpha * x) * w + b (h may be x itself)."""
    _check(x, "residual stream", torch.float32, 2)
    n, d = x.shape
    parts = []
    for t, what in ((a, "mixer output"), (f, "feed-forward output")):
        if t is None:
            parts.append(0)
            continue
        _check(t, what)
        if t.dim() not in (2, 3) or tuple(t.shape[-2:]) != (n, d):
            raise KernelError(f"add_dyt: {what} and the residual stream differ in size")
        parts.append(t.shape[0] if t.dim() == 3 else 1)
    if h is not None:
        _check(h, "norm output", None, 2)
        _check(w, "norm weight", torch.float32, 1)
        _check(b, "norm bias", torch.float32, 1)
        if h.shape != x.shape or w.shape[0] != d or b.shape[0] != d:
            raise KernelError("add_dyt: sizes of the norm disagree")
    rows_lib().call("hos_add_dyt", _ptr(a), dtype_code(a.dtype) if a is not None else 0, parts[0],
                  _ptr(f), dtype_code(f.dtype) if f is not None else 0, parts[1], float(mult), _ptr(x), float(alpha),
                  _ptr(w), _ptr(b), _ptr(h), dtype_code(h.dtype) if h is not None else 0, n, d, _stream())


# ---- a norm after the sum, gated attention with a sink, matrix-state scans (csrc/postnorm.cu, gated_attention.cu,
# ---- state_scan.cu) ----------------------------------------------------------------------------------------------
_mixers: Optional[Library] = None
ACT_LOGISTIC, ACT_X_LOGISTIC = 0, 1


def mixers() -> Library:
    global _mixers
    if _mixers is None:
        _mixers = Library("mixers")
    return _mixers


def scale_add_norm(y: torch.Tensor, alpha: float, x: torch.Tensor, w: torch.Tensor, eps: float,
                   h: Optional[torch.Tensor] = None, w_next: Optional[torch.Tensor] = None, eps_next: float = 0.0) -> None:
    """x <- RMSNorm(alpha * x + y; w, eps).  y: [N, D], or [parts, N, D] float32 partial sums.  With `h`: h = the new x
    in h's type, or, with `w_next`, RMSNorm(x; w_next, eps_next)."""
    _check(x, "residual stream", torch.float32, 2)
    _check(y, "branch output")
    _check(w, "norm weight", torch.float32, 1)
    n, d = x.shape
    if y.dim() not in (2, 3) or tuple(y.shape[-2:]) != (n, d) or w.shape[0] != d:
        raise KernelError("scale_add_norm: sizes disagree")
    if h is not None:
        _check(h, "next input", None, 2)
        if h.shape != x.shape or (w_next is not None and w_next.shape[0] != d):
            raise KernelError("scale_add_norm: sizes of the next input disagree")
    mixers().call("hos_scale_add_norm", _ptr(y), dtype_code(y.dtype), y.shape[0] if y.dim() == 3 else 1, float(alpha),
                  _ptr(x), _ptr(w), float(eps), _ptr(h), dtype_code(h.dtype) if h is not None else 0, _ptr(w_next),
                  float(eps_next), n, d, _stream())


def cast_rows(x: torch.Tensor, h: torch.Tensor) -> None:
    _check(x, "rows", torch.float32)
    _check(h, "rows in the products' type")
    if h.shape != x.shape:
        raise KernelError("cast_rows: sizes disagree")
    mixers().call("hos_cast_rows", _ptr(x), _ptr(h), dtype_code(h.dtype), x.numel(), _stream())


def _at(t: torch.Tensor, col: int):
    """The address of a row-major matrix's column `col`."""
    return ctypes.c_void_p(t.data_ptr() + col * t.element_size())


def group_norm_gate(o: torch.Tensor, w: torch.Tensor, gate: torch.Tensor, gate_col: int, act: int, token_seq,
                    out: torch.Tensor, eps: float, groups: int, group_size: int, out_col: int = 0) -> None:
    """out[n, out_col + (g, :)] = o[n, g, :] / rms * w * act(gate[n, gate_col + g * group_size + :]); w: [group_size]
    (shared by the groups) or [groups * group_size]."""
    _check(o, "mixer output", torch.float32, 2)
    _check(gate, "gate rows", torch.float32, 2)
    _check(w, "norm weight", torch.float32, 1)
    n = o.shape[0]
    _check(out, "gated heads", None, 2)
    if o.shape[1] != groups * group_size or out.shape[0] != n or out_col + o.shape[1] > out.shape[1] or w.shape[0] not in (group_size, groups * group_size) \
            or gate.shape[0] != n or gate_col + groups * group_size > gate.shape[1]:
        raise KernelError("group_norm_gate: sizes disagree")
    shared = 1 if (w.shape[0] == group_size and groups > 1) else 0
    mixers().call("hos_group_norm_gate", _ptr(o), _ptr(w), shared,
                  _at(gate, gate_col), gate.shape[1], int(act), _ptr(token_seq), _at(out, out_col),
                  dtype_code(out.dtype), out.shape[1], float(eps), n, int(groups), int(group_size), _stream())


def skip_gate_norm(o: torch.Tensor, x: torch.Tensor, x_col: int, skip: torch.Tensor, z: torch.Tensor, z_col: int,
                   w: torch.Tensor, eps: float, token_seq, out: torch.Tensor, heads: int, vdim: int, parts: int) -> None:
    """y = (o + skip[head] * x[:, x_col:]) * z logistic(z) with z = z[:, z_col:]; out = y in `parts` equal parts, each divided by
    its own root mean square, times w ([heads * vdim])."""
    for t, what in ((o, "read-outs"), (x, "inputs"), (z, "gates")):
        _check(t, what, torch.float32, 2)
    _check(w, "norm weight", torch.float32, 1)
    _check(skip, "skip factors", torch.float32, 1)
    _check(out, "gated heads", None, 2)
    n, inner = o.shape
    if inner != heads * vdim or out.shape != o.shape or w.shape[0] != inner or skip.shape[0] != heads or inner % parts != 0 \
            or x.shape[0] != n or z.shape[0] != n or x_col + inner > x.shape[1] or z_col + inner > z.shape[1]:
        raise KernelError("skip_gate_norm: sizes disagree")
    mixers().call("hos_skip_gate_norm", _ptr(o), _at(x, x_col), x.shape[1], _ptr(skip), _at(z, z_col), z.shape[1], _ptr(w),
                  float(eps), _ptr(token_seq), _ptr(out), dtype_code(out.dtype), n, int(heads), int(vdim), int(parts), _stream())


# ---- hyper-connections (csrc/hyper.cu) -----------------------------------------------------------------------------

def hyper_norm(x: torch.Tensor, streams: int, y: Optional[torch.Tensor] = None, bias: Optional[torch.Tensor] = None,
               mix: Optional[torch.Tensor] = None, out_w: Optional[torch.Tensor] = None, in_next: Optional[torch.Tensor] = None,
               w: Optional[torch.Tensor] = None, eps: float = 0.0, h: Optional[torch.Tensor] = None) -> None:
    """x: float32 [N, streams * D].  With y ([N, D] of any type, or [parts, N, D] float32 partial sums): x_t <- sum_s
    mix[s, t] x_s + out_w[t] (y + bias).  With h: h = RMSNorm(sum_s in_next[s] x_s; w, eps) (in_next None: ones)."""
    _check(x, "residual streams", torch.float32, 2)
    n, d = x.shape[0], x.shape[1] // streams
    parts = 1
    if x.shape[1] != streams * d:
        raise KernelError("hyper_norm: the row is no whole number of streams")
    if y is not None:
        _check(y, "branch output")
        parts = y.shape[0] if y.dim() == 3 else 1
        if y.dim() not in (2, 3) or tuple(y.shape[-2:]) != (n, d) or mix.shape != (streams, streams) or out_w.shape != (streams,):
            raise KernelError("hyper_norm: sizes of the branch output or its weights disagree")
    for t, shape, what in ((bias, (d,), "bias"), (mix, (streams, streams), "mixing weights"), (out_w, (streams,), "output weights"),
                           (in_next, (streams,), "input weights"), (w, (d,), "norm weight")):
        if t is not None:
            _check(t, what, torch.float32)
            if tuple(t.shape) != shape:
                raise KernelError(f"hyper_norm: {what} of shape {tuple(t.shape)}, {shape} is needed")
    if h is not None:
        _check(h, "norm output", None, 2)
        if tuple(h.shape) != (n, d) or w is None:
            raise KernelError("hyper_norm: sizes of the norm disagree")
    mixers().call("hos_hyper_norm", _ptr(y), dtype_code(y.dtype) if y is not None else 0, parts, _ptr(bias), _ptr(x), int(streams),
                  _ptr(mix), _ptr(out_w), _ptr(in_next), _ptr(w), float(eps), _ptr(h),
                  dtype_code(h.dtype) if h is not None else 0, n, d, _stream())


def stream_sums(x: torch.Tensor, streams: int, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """float32 [n, D]: the sum of the streams of the given rows (all rows where none are given)."""
    _check(x, "residual streams", torch.float32, 2)
    n, d = (x.shape[0] if rows is None else rows.shape[0]), x.shape[1] // streams
    if rows is not None:
        _check(rows, "row indices", torch.int32, 1)
    out = torch.empty((n, d), dtype=torch.float32, device=x.device)
    mixers().call("hos_stream_sums", _ptr(x), _ptr(rows), _ptr(out), n, int(streams), d, _stream())
    return out


def qk_prep(proj: torch.Tensor, bias: Optional[torch.Tensor], q_norm: Optional[torch.Tensor], k_norm: Optional[torch.Tensor],
            eps: float, freq: Optional[torch.Tensor], rot_dims: int, magnitude: float, step, q_out: torch.Tensor,
            cache: PagedKVArgs, n_heads: int, n_kv: int, kd: int, vd: int, norm_whole: bool = False,
            v_first: Optional[torch.Tensor] = None, v_first_col: int = 0, v_mix: float = 0.0, q_maps: int = 1,
            proj_col: int = 0, q_temp=None, style: int = 1, unit_norm: bool = False) -> None:
    """proj: float32 rows whose columns from proj_col on are [q | k | v | ...] (G = n_kv; 0: a call that stores nothing).  Adds the
    biases, norms and rotates the q and k heads, writes q_out float32 [N, H, kd] and stores k, v in the cache.
    norm_whole: one root mean square over all q heads and one over all k heads (weights [H kd], [G kd]).  v_first
    (float32 [N, ld], the values from column v_first_col on): v <- (1 - v_mix) v + v_mix v_first before the store.
    q_maps > 1: a head's kd numbers are q_maps queries, one per attention map over the same key row; q_out is then
    [N, H * q_maps, kd], every query a head of its own that is zero outside its part of the key row.  q_temp = (coef, every): q times
    1 + coef ln(floor((p + 1) / every) + 1) at position p.  style: the rotation's pairing (ROPE_STYLES).  unit_norm: every q and
    k head over its root mean square, without a weight."""
    _check(proj, "projection rows", torch.float32, 2)
    _check(q_out, "queries", torch.float32, 3)
    n = proj.shape[0]
    c = n_heads * kd + n_kv * (kd + vd)
    if q_out.shape != (n, n_heads * q_maps, kd) or proj.shape[1] < proj_col + c:
        raise KernelError("qk_prep: sizes disagree")
    if n_kv and (cache.head_dim != kd or cache.v_dim != vd or cache.n_kv_heads != n_kv):
        raise KernelError("qk_prep: the cache does not fit the keys and values")
    for wn, cols in ((q_norm, n_heads * kd), (k_norm, n_kv * kd)):
        if wn is not None and wn.shape[0] != (cols if norm_whole else kd):
            raise KernelError("qk_prep: a norm weight does not fit the heads")
    vf_ptr, vf_ld = None, 0
    if v_first is not None:
        _check(v_first, "the other layer's values", torch.float32, 2)
        if v_first.shape[0] != n or v_first_col + n_kv * vd > v_first.shape[1]:
            raise KernelError("qk_prep: the other layer's values do not fit this layer's")
        vf_ptr, vf_ld = ctypes.c_void_p(v_first.data_ptr() + 4 * v_first_col), v_first.shape[1]
    coef, every = q_temp if q_temp else (0.0, 0)
    gated_attn_lib().call("hos_qk_prep", _at(proj, proj_col), proj.shape[1], _ptr(bias), _ptr(q_norm), _ptr(k_norm), float(eps), _ptr(freq),
                  int(rot_dims), float(magnitude), _ptr(step.token_pos), _ptr(step.token_seq), _ptr(step.seq_slot),
                  _ptr(q_out), _ptr(cache.k_pages) if n_kv else None, _ptr(cache.v_pages) if n_kv else None,
                  dtype_code(cache.k_pages.dtype), _ptr(cache.page_table), cache.table_stride, cache.ring_pages, n,
                  int(n_heads), int(n_kv), int(kd), int(vd), 1 if norm_whole else 0, vf_ptr, vf_ld, float(v_mix),
                  int(q_maps), float(coef), int(every), int(style), 1 if unit_norm else 0, _stream())


def qkv_conv_store(proj: torch.Tensor, col: int, bias: Optional[torch.Tensor], conv_w: torch.Tensor, conv_state, step, q_out: torch.Tensor,
                   cache: PagedKVArgs, n_heads: int, n_kv: int, kd: int, vd: int, single: bool, q_temp=None) -> None:
    """proj: float32 rows whose C = H kd + G (kd + vd) columns from `col` on are [q | k | v]: every channel passes a short
    convolution over time (conv_w [taps, C]) right after its bias, with its kept inputs conv_state [slots, taps - 1, C]
    (single, only where every sequence brings one token: they move on in this launch; else call conv_keep); queries (times
    their factor, as qk_prep) go to q_out float32 [N, H, kd], keys and values to the cache."""
    _check(proj, "projection rows", torch.float32, 2)
    _check(conv_w, "convolution weights", torch.float32, 2)
    _check(q_out, "queries", torch.float32, 3)
    n, (taps, c) = proj.shape[0], conv_w.shape
    if c != n_heads * kd + n_kv * (kd + vd) or col + c > proj.shape[1] or q_out.shape != (n, n_heads, kd) \
            or (taps > 1 and tuple(conv_state.shape[1:]) != (taps - 1, c)) or (bias is not None and bias.shape[0] < c):
        raise KernelError("qkv_conv_store: sizes disagree")
    if cache.head_dim != kd or cache.v_dim != vd or cache.n_kv_heads != n_kv:
        raise KernelError("qkv_conv_store: the cache does not fit the keys and values")
    coef, every = q_temp if q_temp else (0.0, 0)
    gated_attn_lib().call("hos_qkv_conv_store", _at(proj, col), proj.shape[1], _ptr(bias), _ptr(conv_w), int(taps),
                          _ptr(conv_state) if taps > 1 else None, 1 if single else 0, _ptr(step.token_pos), _ptr(step.token_seq),
                          _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(q_out), _ptr(cache.k_pages), _ptr(cache.v_pages),
                          dtype_code(cache.k_pages.dtype), _ptr(cache.page_table), cache.table_stride, cache.ring_pages, n,
                          int(n_heads), int(n_kv), int(kd), int(vd), float(coef), int(every), _stream())


def diff_combine(a: torch.Tensor, lam: float, mult: float, eps: float, gate: Optional[torch.Tensor], gate_col: int, step,
                 out: torch.Tensor, heads: int, vd: int) -> None:
    """a: float32 [N, heads * 2 * vd], the outputs of a head's two attention maps side by side; out [N, heads * vd] =
    rms_norm_per_head(a1 - lam a2) * mult * logistic(gate[:, gate_col + column])."""
    _check(a, "the maps' outputs", torch.float32, 2)
    n = a.shape[0]
    if a.shape[1] != heads * 2 * vd or out.shape != (n, heads * vd) or \
            (gate is not None and (gate.dtype != torch.float32 or gate_col + heads * vd > gate.shape[1])):
        raise KernelError("diff_combine: sizes disagree")
    gated_attn_lib().call("hos_diff_combine", _ptr(a), float(lam), float(mult), float(eps),
                          ctypes.c_void_p(gate.data_ptr() + gate_col * 4) if gate is not None else None,
                          gate.shape[1] if gate is not None else 0, _ptr(step.token_seq), _ptr(out), dtype_code(out.dtype),
                          n, int(heads), int(vd), _stream())


def gated_attn(q: torch.Tensor, cache: PagedKVArgs, sink: Optional[torch.Tensor], gate: Optional[torch.Tensor],
               gate_col: int, step, out: torch.Tensor, scale: float, chunk: int, window: int, n_splits: int = 1,
               keep_first: int = 0, out_col: int = 0, out_scale: float = 1.0, softcap: float = 0.0) -> None:
    """q: float32 [N, H, kd]; keys and values from the paged cache; out: [N, >= out_col + H * vd], the heads' outputs times
    out_scale from column out_col on.  softcap (0: none): a score s becomes softcap tanh(s / softcap).  gate: float32 rows whose column gate_col + h is head h's gate logit."""
    _check(q, "queries", torch.float32, 3)
    _check(out, "attention output", None, 2)
    n, heads, kd = q.shape
    vd = cache.v_dim
    if out.shape[0] != n or out_col + heads * vd > out.shape[1] or kd != cache.head_dim:
        raise KernelError("gated_attn: sizes disagree")
    part_acc = part_ml = None
    if n_splits > 1:
        part_acc = torch.empty((n, heads, n_splits, vd), dtype=torch.float32, device=q.device)
        part_ml = torch.empty((n, heads, n_splits, 2), dtype=torch.float32, device=q.device)
    gated_attn_lib().call("hos_gated_attn", _ptr(q), _ptr(cache.k_pages), _ptr(cache.v_pages), dtype_code(cache.k_pages.dtype),
                  _ptr(cache.page_table), cache.table_stride, cache.ring_pages, _ptr(sink),
                  ctypes.c_void_p(gate.data_ptr() + gate_col * 4) if gate is not None else None,
                  gate.shape[1] if gate is not None else 0, _ptr(step.token_pos), _ptr(step.token_seq), _ptr(step.seq_slot),
                  _at(out, out_col), dtype_code(out.dtype), out.shape[1], float(out_scale), _ptr(part_acc), _ptr(part_ml),
                  int(n_splits), n, heads,
                  cache.n_kv_heads, kd, vd, float(scale), int(chunk or 0), int(window or 0), int(keep_first or 0), float(softcap), _stream())


def gated_attn_mma(q: torch.Tensor, cache: PagedKVArgs, sink: Optional[torch.Tensor], gate: Optional[torch.Tensor],
                   gate_col: int, step, out: torch.Tensor, scale: float, chunk: int, window: int, n_q_tiles: int,
                   keep_first: int = 0, out_col: int = 0, out_scale: float = 1.0, softcap: float = 0.0) -> bool:
    """The same attention on the tensor cores, for bfloat16 caches and rows that come many to a sequence.  False: the
    sizes are not that kernel's and nothing ran."""
    n, heads, kd = q.shape
    vd = cache.v_dim
    if out.dtype not in (torch.bfloat16, torch.float32) or cache.k_pages.dtype != torch.bfloat16 \
            or out.shape[0] != n or out_col + heads * vd > out.shape[1]:
        return False
    if kd not in (64, 128) or vd not in (64, 128) or q.data_ptr() % 16 or out.data_ptr() % 8 or out.shape[1] % 2 or out_col % 4:
        return False
    gated_attn_lib().call("hos_gated_attn_mma", _ptr(q), _ptr(cache.k_pages), _ptr(cache.v_pages), _ptr(cache.page_table),
                  cache.table_stride, cache.ring_pages, _ptr(sink),
                  ctypes.c_void_p(gate.data_ptr() + gate_col * 4) if gate is not None else None,
                  gate.shape[1] if gate is not None else 0, _ptr(step.cu_seqlens), _ptr(step.token_pos),
                  _ptr(step.token_seq), _ptr(step.seq_slot), _at(out, out_col), 1 if out.dtype == torch.float32 else 0,
                  out.shape[1], float(out_scale), int(step.n_seqs), int(n_q_tiles), heads,
                  cache.n_kv_heads, kd, vd, float(scale), int(chunk or 0), int(window or 0), int(keep_first or 0), float(softcap),
                  _stream())
    return True


def gated_attn_mma_decode(q: torch.Tensor, cache: PagedKVArgs, sink: Optional[torch.Tensor], gate: Optional[torch.Tensor],
                          gate_col: int, step, out: torch.Tensor, scale: float, chunk: int, window: int,
                          n_splits: int = 1, keep_first: int = 0, out_col: int = 0, out_scale: float = 1.0,
                          softcap: float = 0.0) -> bool:
    """Single tokens on the tensor cores: the query heads that share a kv head are the rows of one tile.  False: the
    sizes are not that kernel's and nothing ran."""
    n, heads, kd = q.shape
    vd = cache.v_dim
    if out.dtype not in (torch.bfloat16, torch.float32) or cache.k_pages.dtype != torch.bfloat16 \
            or out.shape[0] != n or out_col + heads * vd > out.shape[1]:
        return False
    if kd not in (64, 128) or vd not in (64, 128) or heads // cache.n_kv_heads > 16 or q.data_ptr() % 16:
        return False
    part_acc = part_ml = None
    if n_splits > 1:
        part_acc = torch.empty((n, heads, n_splits, vd), dtype=torch.float32, device=q.device)
        part_ml = torch.empty((n, heads, n_splits, 2), dtype=torch.float32, device=q.device)
    gate_ptr = ctypes.c_void_p(gate.data_ptr() + gate_col * 4) if gate is not None else None
    gate_ld = gate.shape[1] if gate is not None else 0
    gated_attn_lib().call("hos_gated_attn_mma_decode", _ptr(q), _ptr(cache.k_pages), _ptr(cache.v_pages), _ptr(cache.page_table),
                  cache.table_stride, cache.ring_pages, _ptr(sink), gate_ptr, gate_ld, _ptr(step.token_pos),
                  _ptr(step.token_seq), _ptr(step.seq_slot), _at(out, out_col), 1 if out.dtype == torch.float32 else 0,
                  out.shape[1], float(out_scale), _ptr(part_acc), _ptr(part_ml), int(n_splits), n,
                  heads, cache.n_kv_heads, kd, vd, float(scale), int(chunk or 0), int(window or 0), int(keep_first or 0),
                  float(softcap), _stream())
    if n_splits > 1:
        gated_attn_lib().call("hos_attn_merge", _ptr(part_acc), _ptr(part_ml), int(n_splits), gate_ptr, gate_ld,
                      _ptr(step.token_seq), _at(out, out_col), dtype_code(out.dtype), out.shape[1], float(out_scale), n, heads,
                      vd, _stream())
    return True


segmented_scans = True        # tests switch it off to compare the walk by segments with the whole one


def state_scan(rows: torch.Tensor, q_col: int, k_col: int, v_col: int, silu_on_load: bool, g: torch.Tensor,
               per_token_g: bool, beta: Optional[torch.Tensor], state: torch.Tensor, step, out: torch.Tensor,
               heads: int, key_heads: int, dim: int, vdim: int, rot=None, v_factor: Optional[torch.Tensor] = None,
               channel_g: bool = False, o_mult: float = 1.0) -> None:
    """The matrix-state recurrence over the step's sequences.  v_factor ([N, heads]): with the decay rule, the factor on v.
    channel_g: g is [N, heads * dim], a decay per key channel.  o_mult: a constant on the read-outs.  rot = (freq, rot_dims, style, k_mult): q and k turn with
    their positions and the keys take a factor inside the walk (single-token steps), instead of by rotate_rows before.  rows: float32 [N, ld] holding q, k (key_heads x dim) and
    v (heads x vdim) from the given columns on.  g: [heads] constants, or [N, heads] per token; beta ([N, heads]): the
    delta rule, None: the plain decay rule.  state: [slots, heads, vdim, dim] float32.  out: float32 [N, heads * vdim]."""
    _check(rows, "recurrence inputs", torch.float32, 2)
    _check(state, "recurrent state", torch.float32, 4)
    _check(out, "recurrence output", torch.float32, 2)
    _check(g, "decays", torch.float32)
    n, ld = rows.shape
    if out.shape != (n, heads * vdim) or tuple(state.shape[1:]) != (heads, vdim, dim):
        raise KernelError("state_scan: sizes disagree")
    if channel_g and (tuple(g.shape) != (n, heads * dim) or beta is not None or v_factor is not None or key_heads != heads):
        raise KernelError("state_scan: the decays per key channel do not fit")
    if v_factor is not None:
        _check(v_factor, "factors on v", torch.float32, 2)
        if beta is not None or silu_on_load or tuple(v_factor.shape) != (n, heads):
            raise KernelError("state_scan: factors on v go with the plain decay rule")
    base = rows.data_ptr()
    if rot is not None and (silu_on_load or beta is not None or key_heads != heads):
        raise KernelError("state_scan: the rotation in the walk goes with the plain decay rule on rows as they are")
    rule = 1 if beta is not None else (2 if channel_g else 0)
    second = beta if beta is not None else v_factor
    g_ld = heads * dim if channel_g else (heads if per_token_g else 0)
    seg_len, seg_count, seg_states, seg_decays = 0, 1, None, None
    if rot is None and rule != 1 and segmented_scans:
        seg_len = int(mixers().fn("hos_state_scan_segment")(int(step.n_seqs), int(heads), int(dim), int(vdim), int(step.max_new), rule))
        if seg_len > 0:
            seg_count = -(-int(step.max_new) // seg_len)
            places = int(step.n_seqs) * seg_count * heads
            seg_states = torch.empty(places * vdim * dim, dtype=torch.float32, device=rows.device)
            seg_decays = torch.empty(places * (dim if channel_g else 1), dtype=torch.float32, device=rows.device)
    in_walk = bool(silu_on_load) and beta is None and step.max_new == 1      # single tokens: no launch of its own for it
    if silu_on_load and not in_walk:        # q, k, v lie side by side from q_col on: x logistic(x) in place, once, before the walk
        if not (q_col < k_col < v_col) or v_col + heads * vdim - q_col != 2 * key_heads * dim + heads * vdim:
            raise KernelError("state_scan: q, k, v must lie side by side for the activation")
        mixers().call("hos_act_rows", ctypes.c_void_p(base + 4 * q_col), ld, 2 * key_heads * dim + heads * vdim, n, _stream())
    mixers().call("hos_state_scan", ctypes.c_void_p(base + 4 * q_col), ctypes.c_void_p(base + 4 * k_col),
                  ctypes.c_void_p(base + 4 * v_col), ld, 1 if in_walk else 0, rule, float(o_mult), _ptr(g), g_ld,
                  _ptr(second), heads if second is not None else 0, _ptr(state), _ptr(step.token_pos), _ptr(step.token_seq),
                  _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(out), n, int(step.n_seqs), int(heads), int(key_heads),
                  int(dim), int(vdim), _ptr(rot[0]) if rot else None, int(rot[1]) if rot else 0, int(rot[2]) if rot else 0,
                  float(rot[3]) if rot else 1.0, seg_len, seg_count, _ptr(seg_states), _ptr(seg_decays), _stream(),
                  label="hos_state_scan/channel" if channel_g else ("hos_state_scan/v_factor" if v_factor is not None else None))


def act_rows(rows: torch.Tensor, cols: int) -> None:
    """x logistic(x), in place, on the first `cols` numbers of float32 rows."""
    _check(rows, "projection rows", torch.float32, 2)
    mixers().call("hos_act_rows", _ptr(rows), rows.shape[1], int(cols), rows.shape[0], _stream())


def rotate_rows(rows: torch.Tensor, q_heads: int, k_heads: int, dim: int, freq: Optional[torch.Tensor], rot_dims: int,
                style: int, step, k_mult: float = 1.0) -> None:
    """Rotary positions, in place, on the leading q_heads + k_heads heads of `dim` numbers of float32 rows (the first
    rot_dims numbers of each head, pairing `style`), then the key heads times k_mult."""
    _check(rows, "projection rows", torch.float32, 2)
    if rows.shape[1] < (q_heads + k_heads) * dim:
        raise KernelError("rotate_rows: sizes disagree")
    mixers().call("hos_rotate_rows", _ptr(rows), rows.shape[1], int(q_heads), int(k_heads), int(dim), int(rot_dims),
                  int(style), _ptr(freq), _ptr(step.token_pos), _ptr(step.token_seq), float(k_mult), rows.shape[0], _stream())


def conv_prep(raw: torch.Tensor, conv_w: torch.Tensor, conv_state: torch.Tensor, a_log: torch.Tensor, dt_bias: torch.Tensor,
              step, act: torch.Tensor, beta: torch.Tensor, g: torch.Tensor, heads: int, key_heads: int, dim: int,
              vdim: int, keep_here: bool = False) -> None:
    """raw: float32 [N, ld] = [q | k | v | b | a | ...] projections; conv_w: [C, taps]; conv_state: [slots, taps - 1, C].
    keep_here (only where every sequence brings one token): the kept inputs move on in this launch, conv_keep is not needed."""
    _check(raw, "projection rows", torch.float32, 2)
    _check(conv_w, "convolution weights", torch.float32, 2)
    n, c = raw.shape[0], 2 * key_heads * dim + heads * vdim
    taps = conv_w.shape[1]
    if conv_w.shape[0] != c or raw.shape[1] < c + 2 * heads or act.shape != (n, c) \
            or tuple(conv_state.shape[1:]) != (max(taps - 1, 0), c):
        raise KernelError("conv_prep: sizes disagree")
    mixers().call("hos_conv_prep", _ptr(raw), raw.shape[1], _ptr(conv_w), taps, _ptr(conv_state), _ptr(a_log), _ptr(dt_bias),
                  _ptr(step.token_pos), _ptr(step.token_seq), _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(act),
                  _ptr(beta), _ptr(g), n, int(heads), int(key_heads), int(dim), int(vdim), 1 if keep_here else 0, _stream())


def conv_keep(raw: torch.Tensor, taps: int, conv_state: torch.Tensor, step, channels: int, col: int = 0,
              in_bias: Optional[torch.Tensor] = None) -> None:
    """The last taps - 1 inputs (raw[:, col:col + channels] + in_bias) of every sequence go to the slot's kept inputs."""
    mixers().call("hos_conv_keep", _at(raw, col), raw.shape[1], _ptr(in_bias), int(taps), _ptr(conv_state), _ptr(step.token_pos),
                  _ptr(step.token_seq), _ptr(step.cu_seqlens), _ptr(step.seq_slot), int(step.n_seqs), int(channels),
                  _stream())


def conv_act_rows(raw: torch.Tensor, col: int, conv_w: torch.Tensor, bias: Optional[torch.Tensor], conv_state: torch.Tensor,
                  act: str, step, out: torch.Tensor, single: bool, dt=None, in_bias: Optional[torch.Tensor] = None) -> None:
    """out ([N, C] float32) = act(short convolution of (raw[:, col:col + C] + in_bias) + bias), act "none" or "x_logistic"; conv_w:
    [taps, C]; conv_state: [slots, taps - 1, C] (single, only where every sequence brings one token: the kept inputs move on in this
    launch; else call conv_keep).  dt = (column, dt_bias, a_log, dt_out, g_out): per head, dt_out = softplus(raw + dt_bias) and
    g_out = exp(-exp(a_log) dt) in the same launch."""
    _check(raw, "projection rows", torch.float32, 2)
    _check(conv_w, "convolution weights", torch.float32, 2)
    _check(out, "convolved rows", torch.float32, 2)
    n, (taps, c) = raw.shape[0], conv_w.shape
    if tuple(out.shape) != (n, c) or col + c > raw.shape[1] or tuple(conv_state.shape[1:]) != (taps - 1, c):
        raise KernelError("conv_act_rows: sizes disagree")
    dt_args = (None, None, None, None, None, 0)
    if dt is not None:
        dt_col, dt_bias, a_log, dt_out, g_out = dt
        heads = dt_bias.shape[0]
        for t in (dt_out, g_out):
            _check(t, "step sizes", torch.float32, 2)
            if tuple(t.shape) != (n, heads):
                raise KernelError("conv_act_rows: sizes of the step sizes disagree")
        if dt_col + heads > raw.shape[1] or a_log.shape[0] != heads:
            raise KernelError("conv_act_rows: sizes of the step sizes disagree")
        dt_args = (_at(raw, dt_col), _ptr(dt_bias), _ptr(a_log), _ptr(dt_out), _ptr(g_out), heads)
    mixers().call("hos_conv_act_rows", _at(raw, col), raw.shape[1], _ptr(conv_w), _ptr(in_bias), _ptr(bias), int(taps),
                  _ptr(conv_state) if taps > 1 else None, {"none": 0, "x_logistic": 1}[act], _ptr(step.token_pos), _ptr(step.token_seq),
                  _ptr(step.cu_seqlens), _ptr(step.seq_slot), _ptr(out), n, int(c), 1 if single else 0, *dt_args, _stream())


def channel_decay(rows: torch.Tensor, col: int, rank: int, w: torch.Tensor, b: torch.Tensor, tau: float, out: torch.Tensor) -> None:
    """out ([N, C] float32) = logistic(rows[:, col:col + rank] . w + b)^(1 / tau); w: [rank, C]."""
    _check(rows, "projection rows", torch.float32, 2)
    _check(w, "decay projection", torch.float32, 2)
    _check(b, "decay bias", torch.float32, 1)
    _check(out, "decays", torch.float32, 2)
    n, c = out.shape
    if rows.shape[0] != n or col + rank > rows.shape[1] or tuple(w.shape) != (rank, c) or b.shape[0] != c:
        raise KernelError("channel_decay: sizes disagree")
    mixers().call("hos_channel_decay", _at(rows, col), rows.shape[1], _ptr(w), _ptr(b), int(rank), float(tau), _ptr(out), n, int(c),
                  _stream())
