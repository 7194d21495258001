"""Python faces of the CUDA launchers.  Every function takes CUDA tensors,
launches on the current stream and raises instead of returning a wrong result:
`KernelError` for a launch that failed, `ValueError` for a size a kernel
refuses.  There is no CPU path: a tensor that is not on a GPU is an error."""
from __future__ import annotations

import ctypes
import os
from typing import Optional

import torch

from .build import load_library

F32, BF16 = 0, 1
_DTYPE_TAG = {torch.float32: F32, torch.bfloat16: BF16}


class KernelError(RuntimeError):
    pass


_STATUS_TEXT = {
    -1: "a size this kernel does not take",
    -2: "a dtype this kernel does not take",
    -3: "a pointer or stride that is not aligned as the kernel needs",
    -4: "a bounded wait on the device ran out",
}


class _Counter:
    """How many of the framework's own kernels were launched (the bench reports it)."""
    launches = 0


counter = _Counter()


def _check(status: int, what: str) -> None:
    if status == 0:
        counter.launches += 1
        return
    if status < 0:
        raise ValueError(f"{what}: {_STATUS_TEXT.get(status, f'status {status}')}")
    raise KernelError(f"{what}: CUDA error {status} at launch")


def _tag(t: torch.Tensor) -> int:
    try:
        return _DTYPE_TAG[t.dtype]
    except KeyError:
        raise ValueError(f"kernels take float32 or bfloat16, found {t.dtype}") from None


def _ptr(t: Optional[torch.Tensor]):
    if t is None:
        return ctypes.c_void_p(0)
    if not t.is_cuda:
        raise KernelError("tokenizer_b200 kernels run on a GPU only; got a CPU tensor")
    if not t.is_contiguous():
        raise ValueError("kernels take contiguous tensors")
    return ctypes.c_void_p(t.data_ptr())


_bound_stream = None


def _stream():
    if _bound_stream is not None:
        return _bound_stream
    return ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)


class bound_stream:
    """Within the block every launch goes to the stream that is current at its entry, looked
    up once (asking torch for the current stream costs several microseconds, and a step has a
    few hundred launches).  Nest it anew where the current stream changes (a second stream, a
    graph capture)."""

    def __enter__(self):
        global _bound_stream
        self._outer = _bound_stream
        _bound_stream = ctypes.c_void_p(torch.cuda.current_stream().cuda_stream)
        return self

    def __exit__(self, *exc):
        global _bound_stream
        _bound_stream = self._outer
        return False


_i, _f, _ll = ctypes.c_int, ctypes.c_float, ctypes.c_longlong


class ScratchSpace:
    """Device memory that kernels use beyond their inputs and outputs: the pieces and counters
    of the decode attention, the activation and barrier counters of the fused feed-forward,
    the partial results of the greedy choice.  Counters are zero between launches, and two
    launches that overlap on the device must not share them, so a space belongs to ONE order
    of launches: a model (its forward runs on one stream) and a sampler each own theirs
    (`scratch_scope`), and die with them.  Launches outside any scope (kernel tests) share
    the module's default space, on one stream.  Buffers are made at a shape's first use,
    which is never inside a captured graph: a shape's first step runs plainly."""

    def __init__(self):
        self.decode, self.ffn, self.argmax, self.layer = {}, {}, {}, {}


_default_space = ScratchSpace()
_space = _default_space


class scratch_scope:
    """Within the block, kernels take their scratch from `space`."""

    def __init__(self, space: ScratchSpace):
        self.space = space

    def __enter__(self):
        global _space
        self._outer = _space
        _space = self.space
        return self

    def __exit__(self, *exc):
        global _space
        _space = self._outer
        return False


# ---- the error word ----------------------------------------------------------------
# A wait on the device that runs out does not hang: the kernel sets its library's flag, stores a
# code in one word of mapped pinned host memory and runs to its end WITHOUT the data it waited
# for, so what it wrote is wrong.  Every library gets the word's device address when it is
# loaded; the host reads the word (plain memory, no CUDA call) wherever it has just
# synchronised with the device, and raises.
_LIBRARY_NAMES = {1: "gemm_tcgen05", 2: "attention_tcgen05", 3: "ffn_small_m", 4: "linear_stream",
                  5: "layer_small_m"}
_REASONS = {1: "a wait on a shared-memory barrier ran out", 2: "a wait between blocks ran out"}
_error_word = None          # (ctypes int at the host address, device address)
_registered = {}            # id(library handle) -> handle: libraries that know the word


def _error_word_pointers():
    global _error_word
    if _error_word is None:
        lib = load_library("elementwise.cu")
        host, dev = ctypes.c_void_p(0), ctypes.c_void_p(0)
        status = lib.tokb200_error_word_alloc(ctypes.byref(host), ctypes.byref(dev))
        if status != 0 or not host.value:
            raise KernelError(f"the error word could not be allocated (CUDA error {status})")
        _error_word = (ctypes.c_int.from_address(host.value), dev.value)
    return _error_word


def _load(source: str, defines=()):
    """Load (compile at first use) a library and hand it the error word."""
    lib = load_library(source, defines=defines)
    if id(lib) not in _registered:
        _, dev = _error_word_pointers()
        status = lib.tokb200_set_error_word(ctypes.c_void_p(dev))
        if status != 0:
            raise KernelError(f"{source}: the error word could not be set (CUDA error {status})")
        _registered[id(lib)] = lib
    return lib


def _lib(name):
    return _load(name + ".cu")


def error_code() -> int:
    """The word as it stands (0: no bounded wait has run out); meaningful once the device has
    finished the work in question."""
    return 0 if _error_word is None else int(_error_word[0].value)


def raise_if_error(where: str = "") -> None:
    """Raise KernelError if a bounded wait on the device ran out since the last check.  The
    word and the libraries' flags are cleared, so the next step starts clean.  Costs a read of
    host memory when nothing happened; call it after a synchronisation with the device."""
    code = error_code()
    if code == 0:
        return
    _error_word[0].value = 0
    library, reason = _LIBRARY_NAMES.get(code // 16, f"library {code // 16}"), code % 16
    if reason == 2 and code // 16 == 2:
        text = "a shared-memory base was not aligned as the kernel needs"
    else:
        text = _REASONS.get(reason, f"reason {reason}")
    for lib in _registered.values():          # clear the per-library flags too
        for name in ("tokb200_gemm_tcgen05_error", "tokb200_attention_tcgen05_error",
                     "tokb200_ffn_small_m_error", "tokb200_linear_stream_error",
                     "tokb200_layer_small_m_error"):
            try:
                getattr(lib, name)()
            except AttributeError:
                pass
    raise KernelError(f"{library}: {text}{' (' + where + ')' if where else ''}; the results of the "
                      f"steps since the last check are not valid")


# --------------------------------------------------------------------------- #
def embed(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
    """out[t] = table[ids[t]] * scale, float32."""
    n, hidden = out.shape
    _check(_lib("elementwise").tokb200_embed(
        _ptr(ids), _ptr(table), _i(_tag(table)), _ptr(out), _i(n), _i(hidden),
        _i(table.shape[0]), _f(scale), _stream()), "embed")


def rms_norm(x: torch.Tensor, gain: torch.Tensor, eps: float, out: torch.Tensor,
             delta: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None) -> None:
    """out = norm(x [+ delta]) * gain; with `delta`, x is updated in place.  With
    `rows` (int32), only those rows are read and `out` is dense [len(rows), H]."""
    hidden = x.shape[-1]
    n_rows = out.shape[0]
    if x.dtype != torch.float32 or gain.dtype != torch.float32:
        raise ValueError("rms_norm: the residual stream and the gain are float32")
    if gain.numel() != hidden or out.shape[-1] != hidden:
        raise ValueError("rms_norm: sizes of x, gain and out disagree")
    if delta is not None and rows is not None:
        raise ValueError("rms_norm: a pending residual and a row gather do not combine")
    n_partials, stride = _partials(delta, x)
    _check(_lib("elementwise").tokb200_rms_norm(
        _ptr(x), _ptr(delta), _i(_tag(delta) if delta is not None else F32), _i(n_partials),
        _ll(stride), _ptr(gain),
        _ptr(out), _i(_tag(out)), _ptr(rows), _i(n_rows), _i(hidden), _f(eps), _stream()),
        "rms_norm")


def _partials(delta, x):
    """A pending residual is [T, H], or float32 partial sums [S, T, H] of a
    product that was cut along k; returns (S, elements between partials)."""
    if delta is None or delta.dim() == x.dim():
        if delta is not None and delta.shape != x.shape:
            raise ValueError("the pending residual has another shape than the stream")
        return 1, 0
    if delta.dim() != x.dim() + 1 or delta.shape[1:] != x.shape or delta.dtype != torch.float32:
        raise ValueError("partial sums are float32 [S, T, H]")
    return delta.shape[0], x.numel()


def residual_add(x: torch.Tensor, delta: torch.Tensor) -> None:
    if x.dtype != torch.float32:
        raise ValueError("residual_add: x is float32")
    n_partials, _ = _partials(delta, x)
    _check(_lib("elementwise").tokb200_residual_add(
        _ptr(x), _ptr(delta), _i(_tag(delta)), _i(n_partials), _ll(x.numel()), _stream()),
        "residual_add")


def rope_table(inv_freq: torch.Tensor, n_positions: int):
    half = inv_freq.numel()
    cos = torch.empty((n_positions, half), dtype=torch.float32, device=inv_freq.device)
    sin = torch.empty_like(cos)
    _check(_lib("elementwise").tokb200_rope_table(
        _ptr(inv_freq), _ptr(cos), _ptr(sin), _i(n_positions), _i(half), _stream()), "rope_table")
    return cos, sin


def rope_store(qkv, bias, pos, slot, cos, sin, q_out, k_pool, v_pool, nh, nkv, d, rotary) -> None:
    """Bias, rotation and the write of k and v to their cache slots.  `qkv` is [T, width] or
    float32 partial sums [S, T, width] of a product cut along k (bfloat16 outputs, the whole
    head rotated, head size a multiple of 16)."""
    if qkv.dim() == 3:
        n = qkv.shape[1]
        if qkv.dtype != torch.float32 or qkv.shape[2] != (nh + 2 * nkv) * d or rotary != d or d % 16 or \
                q_out.dtype != torch.bfloat16 or cos.shape[1] != d // 2:
            raise ValueError("rope_store: partial sums are float32 [S, T, width], for bfloat16 "
                             "outputs and a whole-head rotation with head size a multiple of 16")
        _check(_lib("elementwise").tokb200_rope_store_partials(
            _ptr(qkv), _i(qkv.shape[0]), _ptr(bias), _ptr(pos), _ptr(slot), _ptr(cos), _ptr(sin),
            _ptr(q_out), _ptr(k_pool), _ptr(v_pool), _i(n), _i(nh), _i(nkv), _i(d), _stream()),
            "rope_store_partials")
        return
    n = qkv.shape[0]
    if qkv.shape[1] != (nh + 2 * nkv) * d:
        raise ValueError("rope_store: qkv width is not (heads + 2 kv heads) * head_dim")
    if rotary % 2 or (d - rotary) % 2 or rotary > d or cos.shape[1] != rotary // 2:
        raise ValueError(f"rope_store: rotary width {rotary} does not fit head size {d}")
    _check(_lib("elementwise").tokb200_rope_store(
        _ptr(qkv), _ptr(bias), _ptr(pos), _ptr(slot), _ptr(cos), _ptr(sin), _ptr(q_out),
        _ptr(k_pool), _ptr(v_pool), _i(_tag(qkv)), _i(n), _i(nh), _i(nkv), _i(d), _i(rotary),
        _stream()), "rope_store")


# The activation of a feed-forward is a parameter of every kernel that applies one.
ACTIVATIONS = {"silu": 0, "gelu_pytorch_tanh": 1, "relu": 2, "relu_squared": 3}
NO_ACTIVATION = -1


def activation_tag(name: str) -> int:
    try:
        return ACTIVATIONS[name]
    except KeyError:
        raise ValueError(f"the gated kernels know the activations {', '.join(ACTIVATIONS)}; found {name!r}") from None


def product_activation(name: Optional[str]) -> int:
    """The tag of the activation in a plain product's epilogue (None: the product as it is)."""
    return NO_ACTIVATION if name is None else activation_tag(name)


def activate(z: torch.Tensor, activation: str, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """out = act(z), element by element (`out` None: in place)."""
    out = z if out is None else out
    if out.shape != z.shape or out.dtype != z.dtype:
        raise ValueError("activate: out has the shape and type of z")
    _check(_lib("activation").tokb200_activate(
        _ptr(z), _ptr(out), _i(_tag(z)), _i(activation_tag(activation)), _ll(z.numel()), _stream()), "activate")
    return out


def silu_gate(gu: torch.Tensor, out: torch.Tensor, activation: str = "silu") -> None:
    """out[t, i] = act(gu[t, i]) * gu[t, I + i] (the name is from the activation of the
    architecture served; any of `ACTIVATIONS` is taken)."""
    n, inner = out.shape
    if gu.shape[1] != 2 * inner or gu.dtype != out.dtype:
        raise ValueError("silu_gate: input is [T, 2 I], output [T, I], same dtype")
    _check(_lib("elementwise").tokb200_silu_gate(
        _ptr(gu), _ptr(out), _i(_tag(gu)), _i(n), _i(inner), _i(activation_tag(activation)), _stream()),
        "silu_gate")


def _sink(sink, nh):
    """A softmax sink: one float32 per query head, or None."""
    if sink is not None and (sink.dtype != torch.float32 or sink.numel() != nh):
        raise ValueError("attention: a sink is one float32 per query head")
    return _ptr(sink)


def paged_attention_generic(q, k_pool, v_pool, out, block_table, row_req, pos, nh, nkv, d, page,
                            window, scale, sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None,
                            softcap: Optional[float] = None, keep_first: int = 0) -> None:
    """`softcap` (optional, in every attention kernel): a score s becomes softcap * tanh(s / softcap) before
    the softmax.  `chunk` (optional): keys are seen inside chunks of that many positions counted from 0 (a
    query sees the keys of its own chunk up to itself).  `keep_first` (in every attention kernel): the
    sequence's first keys that stay visible although window or chunk have passed them.  `sink` (float32, one per query head): a score without key or value that counts once in
    the softmax's denominator, unscaled.  `v_pool` may be `k_pool` itself (values that are the
    leading lanes of the key rows)."""
    if d > 1024:
        raise ValueError(f"attention: head size {d} is beyond 1024")
    if nh % nkv:
        raise ValueError(f"attention: {nh} heads do not divide into {nkv} groups")
    _check(_lib("attention_generic").tokb200_paged_attention_generic(
        _ptr(q), _ptr(k_pool), _ptr(v_pool), _ptr(out), _i(_tag(q)), _ptr(block_table),
        _i(block_table.shape[1]), _ptr(row_req), _ptr(pos), _i(q.shape[0]), _i(nh), _i(nkv),
        _i(d), _i(page), _i(-1 if window is None else int(window)), _i(0 if chunk is None else int(chunk)), _i(int(keep_first)), _f(scale), _sink(sink, nh), _f(softcap or 0.0), _stream()),
        "paged_attention")


def gemm_f32(a: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor],
             out: torch.Tensor) -> None:
    """out[M,N] = a[M,K] w[N,K]^T (+ bias), true 32-bit."""
    M, K = a.shape
    N = w.shape[0]
    if w.shape[1] != K or out.shape != (M, N):
        raise ValueError("gemm_f32: shapes do not chain")
    for t in (a, w, out):
        if t.dtype != torch.float32:
            raise ValueError("gemm_f32 takes float32")
    _check(_lib("gemm_f32").tokb200_gemm_f32(
        _ptr(a), _ptr(w), _ptr(bias), _ptr(out), _i(M), _i(N), _i(K), _i(K), _i(N), _stream()),
        "gemm_f32")


def sample(logits: torch.Tensor, temperature: Optional[torch.Tensor],
           top_p: Optional[torch.Tensor], uniform: Optional[torch.Tensor],
           out: torch.Tensor) -> None:
    """One token per row of float32 logits; all-None parameters mean greedy."""
    if logits.dtype != torch.float32 or out.dtype != torch.int32:
        raise ValueError("sample: logits are float32, ids int32")
    if temperature is None:
        return argmax(logits, out)
    _check(_lib("sampling").tokb200_sample(
        _ptr(logits), _i(logits.shape[0]), _i(logits.shape[1]), _ptr(temperature), _ptr(top_p),
        _ptr(uniform), _ptr(out), _stream()), "sample")


def prefetch_l2(t: torch.Tensor) -> None:
    """Ask for a tensor's bytes to be brought into L2; returns at once."""
    _check(_lib("elementwise").tokb200_prefetch_l2(
        _ptr(t), _ll(t.numel() * t.element_size()), _stream()), "prefetch_l2")


def advance_decode(ids, drawn, pos, kv_len, row_req, slots, tables, page, history,
                   step_counter) -> None:
    """After a decoding step: the drawn ids become the next inputs and every
    row's position, stored length and cache slot move on by one (on the device)."""
    n = len(slots)
    if n > 32:
        raise ValueError("advance_decode handles up to 32 cache groups")
    slot_ptrs = (ctypes.c_void_p * max(n, 1))(*[t.data_ptr() for t in slots])
    table_ptrs = (ctypes.c_void_p * max(n, 1))(*[t.data_ptr() for t in tables])
    widths = (ctypes.c_int * max(n, 1))(*[t.shape[1] for t in tables])
    _check(_lib("elementwise").tokb200_advance_decode(
        _ptr(ids), _ptr(drawn), _ptr(pos), _ptr(kv_len), _ptr(row_req), _i(n), slot_ptrs,
        table_ptrs, widths, _i(page), _i(ids.shape[0]), _ptr(history), _ptr(step_counter),
        _stream()), "advance_decode")


DECODE_MAX_GROUP = 16


def decode_attention_supported(nh: int, nkv: int, d: int) -> bool:
    """Sizes the split-key decoding kernel takes; others go to the general kernel."""
    return d % 16 == 0 and 16 <= d <= 256 and nh % nkv == 0 and nh // nkv <= DECODE_MAX_GROUP


def decode_attention(q, k_pool, v_pool, out, block_table, row_req, pos, nh, nkv, d, page, window,
                     scale, rows: Optional[torch.Tensor] = None, sink: Optional[torch.Tensor] = None,
                     chunk: Optional[int] = None, softcap: Optional[float] = None, keep_first: int = 0) -> None:
    """Attention for rows of one token each (bfloat16): keys are split over
    blocks and merged; the scratch for the pieces is kept per (device, rows,
    heads, head size) and reused by every layer, which run one after another.  With `rows`
    (int32, -1 for none) only those rows of the batch are served: the single-token rows of a
    step that also brings portions of prompts, which go to the kernels for portions."""
    if q.dtype != torch.bfloat16:
        raise ValueError("decode_attention is the bfloat16 kernel")
    if not decode_attention_supported(nh, nkv, d):
        raise ValueError(f"decode_attention: {nh} heads over {nkv} groups of size {d} is not taken")
    lib = _load("attention_decode.cu", defines=(f"HEAD_DIM={d}",))
    n_rows = q.shape[0] if rows is None else rows.shape[0]
    key = (q.device.index, n_rows, nh, nkv, d)
    if key not in _space.decode:
        lib.tokb200_decode_attention_scratch_floats.restype = ctypes.c_longlong
        floats = lib.tokb200_decode_attention_scratch_floats(_i(n_rows), _i(nh))
        _space.decode[key] = (torch.empty(floats, dtype=torch.float32, device=q.device),
                              torch.zeros(n_rows * nkv, dtype=torch.int32, device=q.device))
    scratch, counters = _space.decode[key]
    _check(lib.tokb200_decode_attention(
        _ptr(q), _ptr(k_pool), _ptr(v_pool), _ptr(out), _ptr(block_table),
        _i(block_table.shape[1]), _ptr(row_req), _ptr(pos), _i(n_rows), _i(nh), _i(nkv), _i(d),
        _i(page), _i(-1 if window is None else int(window)), _i(0 if chunk is None else int(chunk)), _i(int(keep_first)), _f(scale), _ptr(scratch),
        _ptr(counters), _ptr(rows), _sink(sink, nh), _f(softcap or 0.0), _stream()), "decode_attention")


_stream_plans = {}


def linear_stream_supported(M: int, N: int, K: int) -> bool:
    """Sizes the ring-streaming product takes on this device (up to 16 rows, K a multiple of
    32 up to 8192); it pays for matrices of many rows (several tiles of 16 per SM)."""
    if M < 1 or M > 16 or K % 32 or K > 8192:
        return False
    key = (torch.cuda.current_device(), M <= 8, N, K)
    if key not in _stream_plans:
        _stream_plans[key] = bool(_lib("linear_stream").tokb200_linear_stream_supported(_i(M), _i(N), _i(K)))
    return _stream_plans[key]


def linear_stream(x, w, bias, out) -> None:
    """out[M,N] = x w^T (+ bias float32) for up to 16 rows of bfloat16 x and a weight of many
    rows, streamed through shared memory by bulk copies; out is bfloat16 or float32."""
    M, K = x.shape
    N = w.shape[0]
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or w.shape[1] != K:
        raise ValueError("linear_stream: bfloat16 x [M,K] and w [N,K]")
    if tuple(out.shape) != (M, N) or out.dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("linear_stream: out is [M,N] bfloat16 or float32")
    if not linear_stream_supported(M, N, K):
        raise ValueError(f"linear_stream does not take {M} rows with K = {K}")
    _check(_lib("linear_stream").tokb200_linear_stream(
        _ptr(x), _ptr(w), _ptr(bias), _ptr(out), _i(1 if out.dtype == torch.float32 else 0),
        _i(M), _i(N), _i(K), _stream()), "linear_stream")


def linear_stream_check() -> None:
    flag = _lib("linear_stream").tokb200_linear_stream_error()
    if flag:
        raise KernelError("linear_stream: a wait on the device ran out (status %d)" % flag)


_ffn_plans = {}
# compile-time switches of the fused feed-forward's library (a test builds it with short wait limits)
_FFN_DEFINES = ()


def _ffn_lib():
    return _load("ffn_small_m.cu", defines=_FFN_DEFINES)


def ffn_small_m_splits(M: int, hidden: int, inner: int) -> int:
    """Partial sums the fused feed-forward of few rows writes for these sizes on this
    device; 0 when it does not take them (more than 16 rows, hidden not a multiple of
    32, inner not a multiple of 128, too little shared memory)."""
    key = (torch.cuda.current_device(), M <= 8, hidden, inner)
    if M < 1 or M > 16:
        return 0
    if key not in _ffn_plans:
        _ffn_plans[key] = int(_ffn_lib().tokb200_ffn_small_m_splits(_i(M), _i(hidden), _i(inner)))
    return _ffn_plans[key]


def ffn_small_m(x_in, x_out, delta, gain, eps, w_gate_up, w_down, out, activation: str = "silu") -> None:
    """The gated feed-forward of few rows in one kernel: x_out = x_in + delta (delta as
    for rms_norm: [M, H] or float32 partial sums [S, M, H], or None), out [S', M, H] =
    float32 partial sums over k of down(act(gate(h)) * up(h)), h = rms_norm(x_out) * gain.
    `w_gate_up` is in the interleaved row order of `interleave_gate_up`."""
    M, hidden = x_in.shape
    inner = w_down.shape[1]
    if x_in.dtype != torch.float32 or x_out.dtype != torch.float32 or x_out.shape != x_in.shape:
        raise ValueError("ffn_small_m: the residual stream is float32, in and out of one shape")
    if w_gate_up.dtype != torch.bfloat16 or w_down.dtype != torch.bfloat16 or \
            tuple(w_gate_up.shape) != (2 * inner, hidden) or tuple(w_down.shape) != (hidden, inner):
        raise ValueError("ffn_small_m: bfloat16 weights [2 I, H] and [H, I]")
    splits = ffn_small_m_splits(M, hidden, inner)
    if splits == 0:
        raise ValueError(f"ffn_small_m does not take {M} rows of {hidden} with inner size {inner}")
    if tuple(out.shape) != (splits, M, hidden) or out.dtype != torch.float32:
        raise ValueError(f"ffn_small_m: out must be float32 {(splits, M, hidden)}")
    n_partials, stride = _partials(delta, x_in)
    key = (x_in.device.index, inner)
    if key not in _space.ffn:
        _space.ffn[key] = (torch.empty((16, inner), dtype=torch.bfloat16, device=x_in.device),
                           torch.zeros(2, dtype=torch.int32, device=x_in.device))
    act, sync = _space.ffn[key]
    _check(_ffn_lib().tokb200_ffn_small_m(
        _ptr(x_in), _ptr(x_out), _ptr(delta), _i(1 if delta is not None and delta.dtype == torch.float32 else 0),
        _i(n_partials), _ll(stride), _ptr(gain), _f(eps), _ptr(w_gate_up), _ptr(w_down), _ptr(act),
        _ptr(out), _i(M), _i(hidden), _i(inner), _i(activation_tag(activation)), _ptr(sync), _stream()),
        "ffn_small_m")


def ffn_small_m_check() -> None:
    flag = _ffn_lib().tokb200_ffn_small_m_error()
    if flag:
        raise KernelError("ffn_small_m: a wait on the device ran out (status %d)" % flag)


SMALL_M_ROWS = 16     # up to here the streaming kernel leads; above it, the tensor-core tiles


def linear_small_m_supported(M: int, K: int) -> bool:
    return 0 < M <= 64 and K % 8 == 0


def linear_small_m(x, w, bias, out, k_splits: int = 1, activation: Optional[str] = None) -> None:
    """out = act(x w^T (+ bias)) for at most 64 rows of bfloat16 x (`activation` None: no act).  With k_splits > 1
    `out` is float32 [k_splits, M, N]: partial sums that the consumer adds."""
    M, K = x.shape
    N = w.shape[0]
    if not linear_small_m_supported(M, K):
        raise ValueError(f"linear_small_m takes up to 64 rows and K a multiple of 8; got {M} x {K}")
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or w.shape[1] != K:
        raise ValueError("linear_small_m: bfloat16 x [M,K] and w [N,K]")
    want = (M, N) if k_splits == 1 else (k_splits, M, N)
    if tuple(out.shape) != want or (k_splits > 1 and out.dtype != torch.float32):
        raise ValueError(f"linear_small_m: out must be {want}")
    _check(_lib("linear_small_m").tokb200_linear_small_m(
        _ptr(x), _ptr(w), _ptr(bias), _ptr(out), _i(1 if out.dtype == torch.float32 else 0),
        _i(M), _i(N), _i(K), _i(k_splits), _i(product_activation(activation)), _stream()), "linear_small_m")


PREFILL_TILE_ROWS = 64


def prefill_attention_supported(nh: int, nkv: int, d: int) -> bool:
    return d % 16 == 0 and 16 <= d <= 128 and nh % nkv == 0


def prefill_attention(q, k_pool, v_pool, out, block_table, row_req, pos, tiles, n_tiles, nh, nkv,
                      d, page, window, scale, sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None,
                      softcap: Optional[float] = None, keep_first: int = 0) -> None:
    """Attention for portions of prompts (bfloat16).  `tiles` is int32 [n, 2]:
    (first row, rows <= 64) of consecutive rows of one request."""
    if q.dtype != torch.bfloat16:
        raise ValueError("prefill_attention is the bfloat16 kernel")
    if not prefill_attention_supported(nh, nkv, d):
        raise ValueError(f"prefill_attention: {nh} heads over {nkv} groups of size {d} is not taken")
    lib = _load("attention_prefill.cu", defines=(f"HEAD_DIM={d}",))
    _check(lib.tokb200_prefill_attention(
        _ptr(q), _ptr(k_pool), _ptr(v_pool), _ptr(out), _ptr(block_table),
        _i(block_table.shape[1]), _ptr(row_req), _ptr(pos), _ptr(tiles), _i(n_tiles), _i(nh),
        _i(nkv), _i(d), _i(page), _i(-1 if window is None else int(window)), _i(0 if chunk is None else int(chunk)), _i(int(keep_first)), _f(scale), _sink(sink, nh),
        _f(softcap or 0.0), _stream()), "prefill_attention")


def argmax(logits: torch.Tensor, out: torch.Tensor) -> None:
    """Greedy ids (ties keep the lower id): the vocabulary is cut over blocks
    that meet in scratch kept per (device, rows)."""
    n_rows, vocab = logits.shape
    lib = _lib("sampling")
    key = (logits.device.index, n_rows)
    if key not in _space.argmax:
        lib.tokb200_argmax_scratch_bytes.restype = ctypes.c_longlong
        size = lib.tokb200_argmax_scratch_bytes(_i(n_rows))
        _space.argmax[key] = (torch.empty(size, dtype=torch.uint8, device=logits.device),
                              torch.zeros(n_rows, dtype=torch.int32, device=logits.device))
    scratch, counters = _space.argmax[key]
    _check(lib.tokb200_argmax(_ptr(logits), _i(n_rows), _i(vocab), _ptr(out), _ptr(scratch),
                              _ptr(counters), _stream()), "argmax")


def gemm_tcgen05_supported(M: int, N: int, K: int) -> bool:
    return M > 0 and N > 0 and K > 0 and K % 8 == 0


def gemm_tcgen05(a, w, bias, out, block_n: int = 0, activation: Optional[str] = None) -> None:
    """out[M,N] = a[M,K] w[N,K]^T (+ bias) on tcgen05 tensor cores with TMA-fed
    operands; bfloat16 in, bfloat16 or float32 out.  K must be a multiple of 8.  `activation` (bfloat16 out, N a
    multiple of 8): applied in the persistent kernel's epilogue."""
    M, K = a.shape
    N = w.shape[0]
    if a.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or w.shape[1] != K:
        raise ValueError("gemm_tcgen05: bfloat16 a [M,K] and w [N,K]")
    if not gemm_tcgen05_supported(M, N, K):
        raise ValueError(f"gemm_tcgen05: K = {K} must be a multiple of 8")
    if tuple(out.shape) != (M, N) or out.dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("gemm_tcgen05: out is [M,N] bfloat16 or float32")
    if not block_n:
        pitch_ok = N % (4 if out.dtype == torch.float32 else 8) == 0
        if pitch_ok and (M * N >= 128 * 128 * 32 or activation is not None):
            # persistent kernel, TMA-stored output: the wide tile where it divides the work well
            # (with one tile of rows, the narrow tile gives twice the blocks to stream the weights)
            block_n = 1256 if (out.dtype == torch.bfloat16 and N >= 2048 and M > 128) else 1128
        else:
            block_n = 128 if N > 64 else 64
    _check(_lib("gemm_tcgen05").tokb200_gemm_tcgen05(
        _ptr(a), _ptr(w), _ptr(bias), _ptr(out), _i(1 if out.dtype == torch.float32 else 0),
        _i(M), _i(N), _i(K), _i(block_n), _i(product_activation(activation)), _stream()), "gemm_tcgen05")


def gemm_tcgen05_partials(a, w, out) -> None:
    """out[S,M,N] (float32) = partial sums of a[M,K] w[N,K]^T over S pieces of k, for products
    with too few output tiles to fill the device; the consumer adds the pieces in index order."""
    M, K = a.shape
    N = w.shape[0]
    if a.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or w.shape[1] != K:
        raise ValueError("gemm_tcgen05_partials: bfloat16 a [M,K] and w [N,K]")
    if out.dim() != 3 or tuple(out.shape[1:]) != (M, N) or out.dtype != torch.float32:
        raise ValueError("gemm_tcgen05_partials: out is float32 [S,M,N]")
    if K % 8 or N % 4:
        raise ValueError("gemm_tcgen05_partials: K a multiple of 8 and N a multiple of 4")
    _check(_lib("gemm_tcgen05").tokb200_gemm_tcgen05_partials(
        _ptr(a), _ptr(w), _ptr(out), _i(M), _i(N), _i(K), _i(out.shape[0]), _stream()),
        "gemm_tcgen05_partials")


PAIR_PLAIN, PAIR_GATED, PAIR_PARTIALS, PAIR_PLAIN_128 = 0, 1, 2, 3
# TOKB200_GEMM_PAIR=0 keeps every tensor-core product on lone CTAs
_PAIR = os.environ.get("TOKB200_GEMM_PAIR", "1") != "0"


def gemm_tcgen05_pair(a, w, bias, out, kind: int, activation: Optional[str] = None) -> None:
    """The product on pairs of CTAs (two SMs a tile of 256 rows x 256 columns, each loading half
    of the tile's rows of w).  PAIR_PLAIN: out [M,N] bfloat16 (+ bias, then the `activation` where one is named);
    PAIR_GATED: out [M,N/2] bfloat16 = act(gate) * up (silu unless named) for w from `interleave_gate_up`; PAIR_PARTIALS: out [S,M,N]
    float32 partial sums over S pieces of k; PAIR_PLAIN_128: as PAIR_PLAIN with 128-column tiles."""
    M, K = a.shape
    N = w.shape[0]
    if a.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or w.shape[1] != K:
        raise ValueError("gemm_tcgen05_pair: bfloat16 a [M,K] and w [N,K]")
    splits = 1
    if kind == PAIR_PARTIALS:
        if out.dim() != 3 or tuple(out.shape[1:]) != (M, N) or out.dtype != torch.float32 or bias is not None:
            raise ValueError("gemm_tcgen05_pair: partial sums are float32 [S,M,N] without bias")
        splits = out.shape[0]
    elif kind == PAIR_GATED:
        if tuple(out.shape) != (M, N // 2) or out.dtype != torch.bfloat16 or N % 256 or bias is not None:
            raise ValueError("gemm_tcgen05_pair: the gated product is bfloat16 [M,N/2], N a multiple of 256")
    elif kind in (PAIR_PLAIN, PAIR_PLAIN_128):
        if tuple(out.shape) != (M, N) or out.dtype != torch.bfloat16:
            raise ValueError("gemm_tcgen05_pair: out is bfloat16 [M,N]")
    else:
        raise ValueError(f"gemm_tcgen05_pair: kind {kind}")
    if K % 8 or N % (4 if kind == PAIR_PARTIALS else 8):
        raise ValueError("gemm_tcgen05_pair: K a multiple of 8, N of 8 (4 for partial sums)")
    _check(_lib("gemm_tcgen05").tokb200_gemm_tcgen05_pair(
        _ptr(a), _ptr(w), _ptr(bias), _ptr(out), _i(kind), _i(M), _i(N), _i(K), _i(splits),
        _i(activation_tag(activation or "silu") if kind == PAIR_GATED else product_activation(activation)), _stream()),
        "gemm_tcgen05_pair")


def gemm_tcgen05_check() -> None:
    """Raise if a bounded wait inside the tensor-core product ran out since the last check."""
    flag = _lib("gemm_tcgen05").tokb200_gemm_tcgen05_error()
    if flag:
        raise KernelError("gemm_tcgen05: a wait on the device ran out (status %d)" % flag)


def gated_linear_supported(K: int, N: int) -> bool:
    """Gate and up products with the activation folded into the epilogue: the
    stacked weight is laid out in blocks of 128 gate rows + 128 up rows."""
    return K % 8 == 0 and N % 256 == 0


def interleave_gate_up(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """[gate rows 0..127, up rows 0..127, gate rows 128..255, ...]: the layout the
    gated kernels read (both have I rows, I a multiple of 128)."""
    inner, k = gate.shape
    return torch.stack([gate.view(inner // 128, 128, k), up.view(inner // 128, 128, k)], dim=1) \
        .reshape(2 * inner, k).contiguous()


def gated_linear(x, w, out, activation: str = "silu") -> None:
    """out[M, N/2] = act(x Wg^T) * (x Wu^T) for w from `interleave_gate_up`; the activation
    is an epilogue parameter of whichever kernel the row count selects."""
    act = _i(activation_tag(activation))
    M, K = x.shape
    N = w.shape[0]
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or out.dtype != torch.bfloat16:
        raise ValueError("gated_linear is the bfloat16 kernel")
    if not gated_linear_supported(K, N) or w.shape[1] != K or tuple(out.shape) != (M, N // 2):
        raise ValueError("gated_linear: K a multiple of 8, N of 256, out [M, N/2]")
    if M <= SMALL_M_ROWS and _RING and N * K >= RING_ELEMENTS and linear_ring_supported(M, N, K, 1, True):
        linear_ring_gated(x, w, out, activation)
    elif M <= SMALL_M_ROWS:
        _check(_lib("linear_small_m").tokb200_linear_small_m_gated(
            _ptr(x), _ptr(w), _ptr(out), _i(M), _i(N), _i(K), act, _stream()), "gated_linear")
    elif M <= RING_MAX_ROWS and _RING and (M <= 24 or N * K <= 9_000_000) and linear_ring_supported(M, N, K, 1, True):
        # 17 to 32 rows: the ring kernel where it leads a tensor-core tile that is mostly padding
        # followed by the activation's own kernel (us in a captured chain, hidden 896: 11.3 -> 9.0
        # at 17 rows, 13.3 -> 10.6 at 32; hidden 1,536: 24.3 -> 17.5 at 17 rows, but 18.8 -> 20.6 at 32)
        linear_ring_gated(x, w, out, activation)
    elif M <= 64:
        # too few rows to fill the 256-wide gated tiles over the SMs: the plain tensor-core
        # product over the same (interleaved) weight, then the activation on its output
        gu = torch.empty((M, N), dtype=torch.bfloat16, device=x.device)
        gemm_tcgen05(x, w, None, gu)
        _check(_lib("elementwise").tokb200_silu_gate_interleaved(
            _ptr(gu), _ptr(out), _i(M), _i(N // 2), act, _stream()), "silu_gate_interleaved")
    elif M >= 256 and _PAIR:
        # two tiles of rows and more: pairs of CTAs on tiles of 256 rows, each loading half of the
        # weight tile (a sixth fewer cycles than lone CTAs at 2,048 rows)
        _check(_lib("gemm_tcgen05").tokb200_gemm_tcgen05_pair(
            _ptr(x), _ptr(w), None, _ptr(out), _i(PAIR_GATED), _i(M), _i(N), _i(K), _i(1), act, _stream()),
            "gated_linear")
    else:
        _check(_lib("gemm_tcgen05").tokb200_gemm_tcgen05_gated(
            _ptr(x), _ptr(w), _ptr(out), _i(M), _i(N), _i(K), act, _stream()), "gated_linear")


def qkv_rope_small_m_supported(M: int, K: int, d: int, rotary: int, n_out: int = 0) -> bool:
    """Where the fused kernel is the one to use (it takes up to 64 rows).  Up to 32 rows: beyond 16 the streaming product is no longer the fastest on its own, but
    with rotation and cache write in its epilogue it still beats a tile product and a second
    kernel.  Up to 64 rows where the stacked weight is small (`n_out` x K up to two million
    elements: the 0.5B sizes), so that the product's own time hardly matters beside a launch
    saved (batch 64: 1.37 -> 1.28 ms a step)."""
    most = 64 if 0 < n_out * K <= 2_000_000 else 32
    return 0 < M <= most and K % 8 == 0 and d % 16 == 0 and rotary == d


def qkv_rope_small_m(x, w, bias, pos, slot, cos, sin, q_out, k_pool, v_pool, nh, nkv, d) -> None:
    """The stacked q/k/v projection of few rows with bias, rotary encoding and the
    cache write folded into its epilogue (bfloat16; the whole head is rotated)."""
    M, K = x.shape
    if w.shape != ((nh + 2 * nkv) * d, K) or x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16:
        raise ValueError("qkv_rope_small_m: w is the stacked [(heads + 2 kv heads) d, K] weight")
    if not (0 < M <= 64 and K % 8 == 0 and d % 16 == 0 and 2 * cos.shape[1] == d):
        raise ValueError("qkv_rope_small_m: up to 64 rows, K a multiple of 8, the whole head (a multiple of 16) rotated")
    _check(_lib("linear_small_m").tokb200_qkv_rope_small_m(
        _ptr(x), _ptr(w), _ptr(bias), _ptr(pos), _ptr(slot), _ptr(cos), _ptr(sin), _ptr(q_out),
        _ptr(k_pool), _ptr(v_pool), _i(M), _i(nh), _i(nkv), _i(d), _i(K), _stream()),
        "qkv_rope_small_m")


def gemm_qkv_rope_supported(K: int, nh: int, nkv: int, d: int, rotary: int) -> bool:
    """Sizes the tcgen05 q/k/v product with the rotary epilogue takes: head size 64 or 128, the
    whole head rotated, and q and k/v regions of whole 128-column tiles."""
    return K % 8 == 0 and d in (64, 128) and rotary == d and (nh * d) % 128 == 0 and (nkv * d) % 128 == 0


def gemm_qkv_rope(x, w, bias, pos, slot, cos, sin, q_out, k_pool, v_pool, nh, nkv, d) -> None:
    """The stacked q/k/v projection of many rows on tcgen05 with bias, rotary encoding and the
    cache write folded into the epilogue (bfloat16)."""
    M, K = x.shape
    if w.shape != ((nh + 2 * nkv) * d, K) or x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16:
        raise ValueError("gemm_qkv_rope: w is the stacked [(heads + 2 kv heads) d, K] weight")
    if not gemm_qkv_rope_supported(K, nh, nkv, d, 2 * cos.shape[1]) or tuple(q_out.shape) != (M, nh * d):
        raise ValueError("gemm_qkv_rope: sizes it does not take")
    _check(_lib("gemm_tcgen05").tokb200_gemm_tcgen05_qkv_rope(
        _ptr(x), _ptr(w), _ptr(bias), _ptr(pos), _ptr(slot), _ptr(cos), _ptr(sin), _ptr(q_out),
        _ptr(k_pool), _ptr(v_pool), _i(M), _i(nh), _i(nkv), _i(d), _i(K), _stream()), "gemm_qkv_rope")


def qkv_norm_rope_small_m_supported(M: int, K: int, d: int, rotary: int) -> bool:
    """Up to 8 rows (a row a warp; with 16, the norm that every block repeats costs more than
    the launch it saves: 1.03 against 0.92 ms a step), K a multiple of 32 up to 1024."""
    return 0 < M <= 8 and K % 32 == 0 and K <= 1024 and d % 16 == 0 and rotary == d


def qkv_norm_rope_small_m(x, x_out, delta, gain, eps, w, bias, pos, slot, cos, sin, q_out, k_pool,
                          v_pool, nh, nkv, d) -> None:
    """`qkv_rope_small_m` with the residual add and the RMS norm in front computed by the
    kernel itself: x_out = x + delta (delta as for rms_norm: [M, K], float32 partial sums
    [S, M, K], or None), projection of norm(x_out) * gain."""
    M, K = x.shape
    if x.dtype != torch.float32 or x_out.dtype != torch.float32 or x_out.shape != x.shape:
        raise ValueError("qkv_norm_rope_small_m: the residual stream is float32, in and out of one shape")
    if w.shape != ((nh + 2 * nkv) * d, K) or w.dtype != torch.bfloat16:
        raise ValueError("qkv_norm_rope_small_m: w is the stacked [(heads + 2 kv heads) d, K] weight")
    if not qkv_norm_rope_small_m_supported(M, K, d, 2 * cos.shape[1]):
        raise ValueError("qkv_norm_rope_small_m: sizes it does not take")
    n_partials, stride = _partials(delta, x)
    _check(_lib("linear_small_m").tokb200_qkv_norm_rope_small_m(
        _ptr(x), _ptr(x_out), _ptr(delta), _i(1 if delta is not None and delta.dtype == torch.float32 else 0),
        _i(n_partials), _ll(stride), _ptr(gain), _f(eps), _ptr(w), _ptr(bias), _ptr(pos), _ptr(slot),
        _ptr(cos), _ptr(sin), _ptr(q_out), _ptr(k_pool), _ptr(v_pool), _i(M), _i(nh), _i(nkv), _i(d),
        _i(K), _stream()), "qkv_norm_rope_small_m")


WIDE_TILE_ROWS = 128


def attention_tcgen05_supported(nh: int, nkv: int, d: int) -> bool:
    return d in (64, 128) and nh % nkv == 0


def attention_tcgen05(q, k_pool, v_pool, out, block_table, row_req, pos, tiles, n_tiles, nh, nkv, d,
                      page, window, scale, sink: Optional[torch.Tensor] = None, chunk: Optional[int] = None,
                      softcap: Optional[float] = None, keep_first: int = 0) -> None:
    """Attention for portions of prompts on tcgen05 (bfloat16, head size 64 or 128).
    `tiles` is int32 [n, 2]: (first row, rows <= 128) of consecutive rows of one request."""
    if q.dtype != torch.bfloat16:
        raise ValueError("attention_tcgen05 is the bfloat16 kernel")
    if not attention_tcgen05_supported(nh, nkv, d):
        raise ValueError(f"attention_tcgen05: head size {d} is not taken (64 or 128)")
    lib = _load("attention_tcgen05.cu", defines=(f"HEAD_DIM={d}",))
    _check(lib.tokb200_attention_tcgen05(
        _ptr(q), _ptr(k_pool), _ptr(v_pool), _ptr(out), _ptr(block_table),
        _i(block_table.shape[1]), _ptr(row_req), _ptr(pos), _ptr(tiles), _i(n_tiles), _i(nh),
        _i(nkv), _i(d), _i(page), _i(-1 if window is None else int(window)), _i(0 if chunk is None else int(chunk)), _i(int(keep_first)), _f(scale), _sink(sink, nh),
        _f(softcap or 0.0), _stream()), "attention_tcgen05")


def attention_tcgen05_check(d: int) -> None:
    flag = _load("attention_tcgen05.cu", defines=(f"HEAD_DIM={d}",)).tokb200_attention_tcgen05_error()
    if flag:
        raise KernelError("attention_tcgen05: a wait on the device ran out (status %d)" % flag)


# --------------------------------------------------------------------------- #
# a whole decoder layer of few rows in one kernel
class _LayerArgs(ctypes.Structure):
    _fields_ = (
        [(n, ctypes.c_void_p) for n in ("w_qkv", "b_qkv", "w_o", "gain1", "gain2", "w_gu", "w_d", "k_pool",
                                        "v_pool", "k_read", "v_read", "cos_t", "sin_t")] +
        [("eps1", ctypes.c_float), ("eps2", ctypes.c_float), ("scale", ctypes.c_float),
         ("window", ctypes.c_int), ("activation", ctypes.c_int),
         ("x_in", ctypes.c_void_p), ("delta", ctypes.c_void_p), ("delta_is_f32", ctypes.c_int),
         ("n_partials", ctypes.c_int), ("partial_stride", ctypes.c_longlong)] +
        [(n, ctypes.c_void_p) for n in ("x_mid", "x_out", "out", "pos", "slot", "row_req", "block_table")] +
        [("table_stride", ctypes.c_int), ("page", ctypes.c_int)] +
        [(n, ctypes.c_void_p) for n in ("q_buf", "att_part", "att_count", "att_out", "o_part", "act", "sync")] +
        [(n, ctypes.c_int) for n in ("M", "H", "I", "nh", "nkv", "d")] +
        [("stamps", ctypes.c_void_p), ("next_w_qkv", ctypes.c_void_p), ("next_gain1", ctypes.c_void_p),
         ("next_b_qkv", ctypes.c_void_p), ("repeat", ctypes.c_int)])


LAYER_HEAD_DIMS = (64, 128)
LAYER_MAX_ROWS = 32
LAYER_MAX_SPLITS = 32
_layer_plans = {}
# compile-time switches of the layer kernel's library (a test builds it with short wait limits)
_LAYER_DEFINES = ()


def _layer_lib(d: int):
    return _load("layer_small_m.cu", defines=(f"HEAD_DIM={d}",) + tuple(_LAYER_DEFINES))


def layer_small_m_splits(M: int, hidden: int, inner: int, nh: int, nkv: int, d: int):
    """(partial sums of the feed-forward, partial sums of the output projection) that the
    whole-layer kernel of few rows writes for these sizes on this device; (0, 0) when it does
    not take them (more than 32 rows, a head size it is not built for, hidden not a multiple
    of 32 or beyond 4096, inner not a multiple of 128, groups of more than 16 heads, too
    little shared memory for its ring)."""
    if M < 1 or M > LAYER_MAX_ROWS or d not in LAYER_HEAD_DIMS:
        return 0, 0
    key = (torch.cuda.current_device(), (M > 8) + (M > 16), hidden, inner, nh, nkv, d)
    if key not in _layer_plans:
        o_splits = ctypes.c_int(0)
        down = int(_layer_lib(d).tokb200_layer_small_m_splits(_i(M), _i(hidden), _i(inner), _i(nh), _i(nkv),
                                                              ctypes.byref(o_splits)))
        _layer_plans[key] = (down, int(o_splits.value))
    return _layer_plans[key]


def layer_small_m(x_in, delta, x_mid, x_out, out, gain1, eps1, w_qkv, b_qkv, pos, slot, row_req, block_table,
                  cos, sin, k_pool, v_pool, writes: bool, w_o, gain2, eps2, w_gate_up, w_down, nh: int,
                  nkv: int, d: int, page: int, window, scale: float, activation: str = "silu",
                  stamps: Optional[torch.Tensor] = None, next_layer=None, repeat: int = 1) -> None:
    """One pre-norm decoder layer for up to 32 rows of one token each (bfloat16): x_mid = x_in +
    delta; attention (q/k/v with bias, rotary encoding, cache write when `writes`, softmax over
    the paged keys) of rms_norm(x_mid) * gain1; x_out = x_mid + its output projection; out
    [S, M, H] = float32 partial sums over k of the gated feed-forward of rms_norm(x_out) * gain2.
    `delta` as for rms_norm ([M, H], float32 partial sums [S, M, H], or None); `w_gate_up` in the
    row order of `interleave_gate_up`; `out` has `layer_small_m_splits(...)[0]` planes.  `stamps`
    (int64 [blocks, 16], for profiling) receives the time in ns at which each block passes each phase;
    `next_layer` = (q/k/v weight of the same shape, first gain, q/k/v bias or None) of the layer that
    runs next: what that layer's kernel starts with is brought into L2 ahead."""
    M, hidden = x_in.shape
    inner = w_down.shape[1]
    down_splits, o_splits = layer_small_m_splits(M, hidden, inner, nh, nkv, d)
    if down_splits == 0:
        raise ValueError(f"layer_small_m does not take {M} rows of {hidden}, inner {inner}, {nh}/{nkv} heads of {d}")
    for t in (x_in, x_mid, x_out):
        if t.dtype != torch.float32 or tuple(t.shape) != (M, hidden):
            raise ValueError("layer_small_m: the residual stream is float32 [M, H], in, middle and out")
    if tuple(out.shape) != (down_splits, M, hidden) or out.dtype != torch.float32:
        raise ValueError(f"layer_small_m: out must be float32 {(down_splits, M, hidden)}")
    q_width = nh * d
    if w_qkv.dtype != torch.bfloat16 or tuple(w_qkv.shape) != ((nh + 2 * nkv) * d, hidden) or \
            tuple(w_o.shape) != (hidden, q_width) or tuple(w_gate_up.shape) != (2 * inner, hidden) or \
            tuple(w_down.shape) != (hidden, inner) or w_o.dtype != torch.bfloat16 or \
            w_gate_up.dtype != torch.bfloat16 or w_down.dtype != torch.bfloat16:
        raise ValueError("layer_small_m: bfloat16 weights [(nh + 2 nkv) d, H], [H, nh d], [2 I, H], [H, I]")
    if cos.shape[1] != d // 2 or k_pool.dtype != torch.bfloat16:
        raise ValueError("layer_small_m: the whole head is rotated, and the cache is bfloat16")
    n_partials, stride = _partials(delta, x_in)
    key = (x_in.device.index, M, hidden, inner, nh, nkv, d)
    if key not in _space.layer:
        dev = x_in.device
        _space.layer[key] = dict(
            q_buf=torch.empty((M, q_width), dtype=torch.bfloat16, device=dev),
            att_part=torch.empty((M, nh, LAYER_MAX_SPLITS, d + 2), dtype=torch.float32, device=dev),
            att_count=torch.zeros(M * nkv, dtype=torch.int32, device=dev),
            att_out=torch.zeros((M, q_width), dtype=torch.bfloat16, device=dev),
            o_part=torch.empty((o_splits, M, hidden), dtype=torch.float32, device=dev),
            act=torch.empty((LAYER_MAX_ROWS, inner), dtype=torch.bfloat16, device=dev),
            sync=torch.zeros(2, dtype=torch.int32, device=dev))
    sc = _space.layer[key]

    def ptr(t):
        return _ptr(t).value

    args = _LayerArgs(
        w_qkv=ptr(w_qkv), b_qkv=ptr(b_qkv), w_o=ptr(w_o), gain1=ptr(gain1), gain2=ptr(gain2),
        w_gu=ptr(w_gate_up), w_d=ptr(w_down), k_pool=ptr(k_pool) if writes else None,
        v_pool=ptr(v_pool) if writes else None, k_read=ptr(k_pool), v_read=ptr(v_pool), cos_t=ptr(cos),
        sin_t=ptr(sin), eps1=eps1, eps2=eps2, scale=scale, window=-1 if window is None else int(window),
        activation=activation_tag(activation), x_in=ptr(x_in), delta=ptr(delta),
        delta_is_f32=1 if delta is not None and delta.dtype == torch.float32 else 0, n_partials=n_partials,
        partial_stride=stride, x_mid=ptr(x_mid), x_out=ptr(x_out), out=ptr(out), pos=ptr(pos),
        slot=ptr(slot) if writes else None, row_req=ptr(row_req), block_table=ptr(block_table),
        table_stride=block_table.shape[1], page=page, q_buf=ptr(sc["q_buf"]), att_part=ptr(sc["att_part"]),
        att_count=ptr(sc["att_count"]), att_out=ptr(sc["att_out"]), o_part=ptr(sc["o_part"]),
        act=ptr(sc["act"]), sync=ptr(sc["sync"]), M=M, H=hidden, I=inner, nh=nh, nkv=nkv, d=d,
        stamps=ptr(stamps), repeat=repeat)
    if next_layer is not None and next_layer[0].shape == w_qkv.shape:
        args.next_w_qkv, args.next_gain1 = ptr(next_layer[0]), ptr(next_layer[1])
        args.next_b_qkv = ptr(next_layer[2])
    _check(_layer_lib(d).tokb200_layer_small_m(ctypes.byref(args), _stream()), "layer_small_m")


def layer_small_m_check(d: int) -> None:
    flag = _layer_lib(d).tokb200_layer_small_m_error()
    if flag:
        raise KernelError("layer_small_m: a wait on the device ran out (status %d)" % flag)


# ---- few rows, a large weight: one block a multiprocessor streams it through rings in shared memory ----
RING_ELEMENTS = 13_000_000     # from this many weight elements on (26 MB) the ring kernel leads the one with plain loads
RING_MAX_ROWS = 32
_RING = os.environ.get("TOKB200_RING", "1") != "0"     # TOKB200_RING=0: large weights on linear_small_m too
_ring_plans = {}


def linear_ring_supported(M: int, N: int, K: int, k_splits: int = 1, gated: bool = False) -> bool:
    """Sizes `linear_ring` / its gated form take on this device (up to 32 rows, K a multiple of 8 with at
    least 512 per piece of k, x's piece of k and the rings within a block's shared memory)."""
    if not (0 < M <= RING_MAX_ROWS and N > 0 and K > 0 and K % 8 == 0):
        return False
    key = (torch.cuda.current_device(), (M > 8) + (M > 16), N, K, k_splits, gated)
    if key not in _ring_plans:
        _ring_plans[key] = bool(_lib("linear_ring").tokb200_linear_ring_supported(
            _i(M), _i(N), _i(K), _i(k_splits), _i(1 if gated else 0)))
    return _ring_plans[key]


def linear_ring_splits(M: int, N: int, K: int, sms: int) -> int:
    """Pieces of k for a product whose consumer takes partial sums: the count (1 to 8) whose units of
    work (row tiles x pieces) divide most evenly over one block a multiprocessor, among those the
    kernel takes; 0 if it takes none."""
    tiles = -(-N // 16)
    best, best_waste = 0, None
    for s in range(1, 9):
        if not linear_ring_supported(M, N, K, s):
            continue
        units = tiles * s
        rounds = -(-units // sms)
        waste = rounds * sms / units
        if best_waste is None or waste < best_waste - 0.02:
            best, best_waste = s, waste
    return best


def linear_ring(x, w, bias, out, k_splits: int = 1, activation: Optional[str] = None) -> None:
    """out = act(x @ w.T (+ bias)) (`activation` None: no act) for up to 16 rows and a large weight (bfloat16 in; out [M,N]
    bfloat16/float32, or float32 partial sums [k_splits, M, N] without bias)."""
    M, K = x.shape
    N = w.shape[0]
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or w.shape[1] != K:
        raise ValueError("linear_ring: bfloat16 x [M,K] and w [N,K]")
    if not linear_ring_supported(M, N, K, k_splits):
        raise ValueError(f"linear_ring does not take {M} rows, {N} x {K}, {k_splits} pieces of k")
    if k_splits > 1:
        if tuple(out.shape) != (k_splits, M, N) or out.dtype != torch.float32 or bias is not None:
            raise ValueError("linear_ring: partial sums are float32 [S,M,N] without bias")
    elif tuple(out.shape) != (M, N) or out.dtype not in (torch.bfloat16, torch.float32):
        raise ValueError("linear_ring: out is [M,N] bfloat16 or float32")
    _check(_lib("linear_ring").tokb200_linear_ring(
        _ptr(x), _ptr(w), _ptr(bias), _ptr(out), _i(1 if out.dtype == torch.float32 else 0), _i(M), _i(N), _i(K),
        _i(k_splits), _i(product_activation(activation)), _stream()), "linear_ring")


def linear_ring_gated(x, w, out, activation: str = "silu") -> None:
    """out[M, N/2] = act(x Wg^T) * (x Wu^T) for w from `interleave_gate_up`, up to 16 rows, a large weight."""
    M, K = x.shape
    N = w.shape[0]
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or out.dtype != torch.bfloat16 or \
            w.shape[1] != K or tuple(out.shape) != (M, N // 2):
        raise ValueError("linear_ring_gated: bfloat16 x [M,K], w [N,K], out [M,N/2]")
    if not linear_ring_supported(M, N, K, 1, True):
        raise ValueError(f"linear_ring_gated does not take {M} rows, {N} x {K}")
    _check(_lib("linear_ring").tokb200_linear_ring_gated(
        _ptr(x), _ptr(w), _ptr(out), _i(M), _i(N), _i(K), _i(activation_tag(activation)), _stream()),
        "linear_ring_gated")


# ---- a gated recurrence, row-wise activations and gates, the kernels around a cached latent ----
def _ld(t: torch.Tensor) -> int:
    """Elements between the rows of a matrix whose rows are dense (a column slice of a wider one)."""
    if t.dim() != 2 or t.stride(1) != 1:
        raise ValueError("a matrix with dense rows is expected")
    return t.stride(0)


def _sliced_ptr(t: torch.Tensor):
    if not t.is_cuda:
        raise KernelError("tokenizer_b200 kernels run on a GPU only; got a CPU tensor")
    return ctypes.c_void_p(t.data_ptr())


def min_gru_scan(proj: torch.Tensor, z_at: int, u_at: int, g_at: int, width: int, state: torch.Tensor,
                 q_start: torch.Tensor, state_slot: torch.Tensor, longest: int, out: torch.Tensor,
                 bias: Optional[torch.Tensor] = None) -> None:
    """The minGRU recurrence over a step's rows (see csrc/recurrence.cu).  `proj` [T, N] holds the
    three pre-activations in column ranges starting at z_at, u_at, g_at (`bias`, float32 [N]: the
    product's bias, added here); `state` float32 [slots, width] is read and written in place; `out`
    [T, width] dense."""
    if state.dtype != torch.float32 or state.shape[-1] != width or tuple(out.shape) != (proj.shape[0], width):
        raise ValueError("min_gru_scan: state is float32 [slots, width], out [T, width]")
    if max(z_at, u_at, g_at) + width > proj.shape[1] or (bias is not None and (
            bias.dtype != torch.float32 or bias.numel() < max(z_at, u_at, g_at) + width)):
        raise ValueError("min_gru_scan: the column ranges leave the projection (or its bias)")
    _check(_lib("recurrence").tokb200_min_gru_scan(
        _sliced_ptr(proj), _i(_tag(proj)), _ptr(bias), _i(_ld(proj)), _i(z_at), _i(u_at), _i(g_at), _i(width), _ptr(state),
        _ptr(q_start), _ptr(state_slot), _i(q_start.shape[0] - 1), _i(longest), _ptr(out), _i(_tag(out)),
        _stream()), "min_gru_scan")


def poly_norm(z: torch.Tensor, coeff: torch.Tensor, eps: float, out: torch.Tensor,
              bias: Optional[torch.Tensor] = None) -> None:
    """out = a N(v) + b N(v^2) + c N(v^3) + e per row, v = z (+ bias, float32 [n]), N(v) = v /
    sqrt(mean(v^2) + eps); `coeff` float32 [4] = (a, b, c, e) on the device; `z` may be a column
    slice of a wider matrix."""
    n_rows, n = z.shape
    if coeff.dtype != torch.float32 or coeff.numel() != 4 or tuple(out.shape) != (n_rows, n) or \
            (bias is not None and (bias.dtype != torch.float32 or bias.numel() != n)):
        raise ValueError("poly_norm: four float32 numbers, out of z's shape, a float32 bias of z's width")
    _check(_lib("activation").tokb200_poly_norm(
        _sliced_ptr(z), _i(_tag(z)), _sliced_ptr(bias) if bias is not None else _ptr(None), _i(_ld(z)), _ptr(coeff), _ptr(out), _i(_tag(out)), _i(n_rows), _i(n),
        _f(eps), _stream()), "poly_norm")


def gated_delta(y: torch.Tensor, bias: Optional[torch.Tensor], pre: torch.Tensor, out: torch.Tensor,
                pre_bias: Optional[torch.Tensor] = None) -> None:
    """out (float32 [T, H]) = (y + bias) * sigmoid(pre + pre_bias): `y` is [T, H] or float32 partial
    sums [S, T, H]; `pre` [T, H] may be a column slice of a wider matrix; the biases are float32 [H]."""
    n_rows, hidden = out.shape
    if out.dtype != torch.float32 or tuple(pre.shape) != (n_rows, hidden):
        raise ValueError("gated_delta: out is float32 [T, H], the gate's pre-activation [T, H]")
    n_partials, stride = _partials(y, out)
    _check(_lib("activation").tokb200_gated_delta(
        _ptr(y), _i(_tag(y)), _i(n_partials), _ll(stride), _ptr(bias), _sliced_ptr(pre), _i(_tag(pre)),
        _sliced_ptr(pre_bias) if pre_bias is not None else _ptr(None), _i(_ld(pre)), _ptr(out), _i(n_rows), _i(hidden), _stream()), "gated_delta")


def gated_add_rms_norm(x: torch.Tensor, y: torch.Tensor, bias: Optional[torch.Tensor], pre: torch.Tensor,
                       pre_bias: Optional[torch.Tensor], gain: torch.Tensor, eps: float, out: torch.Tensor) -> None:
    """x += (y + bias) * sigmoid(pre + pre_bias) in place (x float32 [T, H]; y, bias, pre, pre_bias as
    for `gated_delta`), then out = x / sqrt(mean(x^2) + eps) * gain: the gate, the residual add and the
    norm that follows in one pass over the row."""
    n_rows, hidden = x.shape
    if x.dtype != torch.float32 or gain.dtype != torch.float32 or gain.numel() != hidden or \
            tuple(out.shape) != (n_rows, hidden) or tuple(pre.shape) != (n_rows, hidden):
        raise ValueError("gated_add_rms_norm: x float32 [T, H], a float32 gain of H, out and the gate [T, H]")
    n_partials, stride = _partials(y, x)
    _check(_lib("activation").tokb200_gated_add_rms_norm(
        _ptr(x), _ptr(y), _i(_tag(y)), _i(n_partials), _ll(stride), _ptr(bias), _sliced_ptr(pre), _i(_tag(pre)),
        _sliced_ptr(pre_bias) if pre_bias is not None else _ptr(None), _i(_ld(pre)), _ptr(gain), _f(eps),
        _ptr(out), _i(_tag(out)), _i(n_rows), _i(hidden), _stream()), "gated_add_rms_norm")


def latent_prepare(proj: torch.Tensor, q_at: int, q_rank: int, c_at: int, kv_rank: int, rot_dim: int,
                   rot_dims: int, q_gain, c_gain, eps: float, inv_freq, pos, row_req, slot, q_latent, pool) -> None:
    """From one projection's rows: the normed query latent (dense, `q_latent` [T, q_rank]) and the
    token's cache row in `pool` [slots, 1, row]: the normed key/value latent and, behind it, the
    positional key part rotated at the token's position (see csrc/latent.cu).  `slot` None: no
    cache write."""
    if pool.dtype != q_latent.dtype or tuple(q_latent.shape) != (proj.shape[0], q_rank):
        raise ValueError("latent_prepare: the query latent is [T, q_rank] in the cache's type")
    _check(_lib("latent").tokb200_latent_prepare(
        _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(q_at), _i(q_rank), _i(c_at), _i(kv_rank), _i(rot_dim),
        _i(rot_dims), _ptr(q_gain), _ptr(c_gain), _f(eps), _ptr(inv_freq), _ptr(pos), _ptr(row_req), _ptr(slot),
        _ptr(q_latent), _ptr(pool), _i(pool.shape[-1] * pool.shape[-2]), _i(_tag(pool)), _i(proj.shape[0]),
        _stream()), "latent_prepare")


def rotate_interleaved(x: torch.Tensor, heads: int, lane0: int, dims: int, inv_freq, pos, row_req) -> None:
    """Rotary encoding in place on lanes lane0 .. lane0 + dims of every head of x [T, heads * row],
    lane 2i paired with lane 2i + 1, angle = position * inv_freq[i] (float32)."""
    n_rows, width = x.shape
    if width % heads:
        raise ValueError("rotate_interleaved: the row does not divide into the heads")
    _check(_lib("latent").tokb200_rotate_interleaved(
        _ptr(x), _i(_tag(x)), _i(heads), _i(width // heads), _i(lane0), _i(dims), _ptr(inv_freq), _ptr(pos),
        _ptr(row_req), _i(n_rows), _stream()), "rotate_interleaved")


# ---- layer norm, the stream's steps around normed sublayer outputs ----
def layer_norm(x: torch.Tensor, gain: torch.Tensor, bias: torch.Tensor, eps: float, out: torch.Tensor,
               rows: Optional[torch.Tensor] = None) -> None:
    """out = (x - mean) / sqrt(var + eps) * gain + bias over the last axis of x (float32 [T, H]); with
    `rows` (int32) only those rows are read and `out` is dense [len(rows), H]."""
    hidden = x.shape[-1]
    if x.dtype != torch.float32 or gain.dtype != torch.float32 or bias.dtype != torch.float32 or \
            gain.numel() != hidden or bias.numel() != hidden or out.shape[-1] != hidden:
        raise ValueError("layer_norm: x, gain and bias are float32 of one width")
    _check(_lib("layer_norm").tokb200_layer_norm(
        _ptr(x), _ptr(gain), _ptr(bias), _ptr(out), _i(_tag(out)), _ptr(rows), _i(out.shape[0]), _i(hidden),
        _f(eps), _stream()), "layer_norm")


def _term(term, like):
    """(pointer, dtype tag, partial sums, their distance, scale) of one scaled term of a sublayer's
    output: (tensor [T, H] or float32 partial sums [S, T, H], scale), or None."""
    if term is None:
        return [_ptr(None), _i(F32), _i(1), _ll(0), _f(0.0)]
    y, scale = term
    n_partials, stride = _partials(y, like)
    return [_ptr(y), _i(_tag(y)), _i(n_partials), _ll(stride), _f(scale)]


def post_norm_add(x: torch.Tensor, terms, gain, bias, eps: float, next_gain=None, next_bias=None,
                  next_eps: float = 0.0, out: Optional[torch.Tensor] = None, rms: bool = False,
                  next_rms: bool = False) -> None:
    """x += LN(sum of the scaled terms) * gain + bias in place (x float32 [T, H]; `terms`: one or two
    (tensor, scale)); with `out`, also out = LN(x) * next_gain + next_bias of the new x.  `rms` / `next_rms`:
    that norm is the RMS form, y / sqrt(mean(y^2) + eps) * gain, and its bias may be None."""
    n_rows, hidden = x.shape
    if x.dtype != torch.float32 or not 1 <= len(terms) <= 2 or gain.numel() != hidden or \
            (bias is None and not rms) or (bias is not None and bias.numel() != hidden):
        raise ValueError("post_norm_add: x float32 [T, H], one or two terms, gain and bias of H")
    if out is not None and (next_gain is None or (next_bias is None and not next_rms) or
                            tuple(out.shape) != (n_rows, hidden)):
        raise ValueError("post_norm_add: the norm behind the add needs gain, bias and out [T, H]")
    args = _term(terms[0], x) + _term(terms[1] if len(terms) > 1 else None, x)
    _check(_lib("layer_norm").tokb200_post_norm_add(
        _ptr(x), *args, _ptr(gain), _ptr(bias), _f(eps), _ptr(next_gain), _ptr(next_bias), _f(next_eps),
        _ptr(out), _i(_tag(out) if out is not None else F32), _i(n_rows), _i(hidden), _i(int(rms)), _i(int(next_rms)),
        _stream()), "post_norm_add")


def scaled_sum(terms, out: torch.Tensor) -> None:
    """out (float32 [T, H]) = sum of one or two scaled terms ((tensor or partial sums, scale))."""
    if out.dtype != torch.float32 or not 1 <= len(terms) <= 2:
        raise ValueError("scaled_sum: out is float32, one or two terms")
    args = _term(terms[0], out) + _term(terms[1] if len(terms) > 1 else None, out)
    _check(_lib("layer_norm").tokb200_scaled_sum(*args, _ptr(out), _ll(out.numel()), _stream()), "scaled_sum")


def stream_inject(x: torch.Tensor, other: Optional[torch.Tensor], vector: Optional[torch.Tensor]) -> None:
    """x[t] += other[t] + vector, each where given (float32)."""
    n_rows, hidden = x.shape
    if x.dtype != torch.float32 or (other is not None and (other.dtype != torch.float32 or other.shape != x.shape)) or \
            (vector is not None and (vector.dtype != torch.float32 or vector.numel() != hidden)):
        raise ValueError("stream_inject: float32 [T, H] and a float32 vector of H")
    _check(_lib("layer_norm").tokb200_stream_inject(_ptr(x), _ptr(other), _ptr(vector), _i(n_rows), _i(hidden),
                                                    _stream()), "stream_inject")


# ---- the gated delta rule ----
def gdn_padded_dim(dim: int) -> int:
    """Rows of a head's state column as the recurrence keeps it (dim rounded up to what its threads
    hold: a power of two times 8 rows for heads of up to 32 lanes, 16 up to 128, 32 beyond); 0: a size it
    does not take."""
    return int(_lib("delta_rule").tokb200_gdn_padded_dim(_i(dim)))


def gdn_prepare(proj: torch.Tensor, qkv_at: int, b_at: int, a_at: int, groups: int, heads: int, dim: int, vdim: int,
                taps: int, conv_w, a_log, dt_bias, state: torch.Tensor, conv_off: int, row_req, q_start, state_slot,
                qkv_out: torch.Tensor, bg_out: torch.Tensor) -> None:
    """Short convolution + silu of q, k, v (from `proj`'s columns qkv_at ..), unit vectors for q (times
    dim^-1/2) and k, beta = sigmoid(proj[b_at ..]) and the decay exp(-exp(a_log) softplus(proj[a_at ..] +
    dt_bias)) and q . k of every group -> `qkv_out` float32 [T, channels], `bg_out` float32 [T, 2 heads + groups]
    (beta, the decay, q . k); then the convolution's
    kept inputs in `state` (float32 [slots, n], at `conv_off` in a slot) move on by the step's rows."""
    channels = 2 * groups * dim + heads * vdim
    n = proj.shape[0]
    if state.dtype != torch.float32 or state.dim() != 2 or tuple(qkv_out.shape) != (n, channels) or \
            tuple(bg_out.shape) != (n, 2 * heads + groups) or qkv_out.dtype != torch.float32 or bg_out.dtype != torch.float32 or \
            conv_w.numel() != channels * taps or conv_off + (taps - 1) * channels > state.shape[1]:
        raise ValueError("gdn_prepare: sizes of the state, the taps or the outputs disagree")
    _check(_lib("delta_rule").tokb200_gdn_prepare(
        _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(qkv_at), _i(b_at), _i(a_at), _i(groups), _i(heads), _i(dim),
        _i(vdim), _i(taps), _ptr(conv_w), _ptr(a_log), _ptr(dt_bias), _ptr(state), _ll(state.shape[1]), _i(conv_off),
        _ptr(row_req), _ptr(q_start), _ptr(state_slot), _i(n), _i(q_start.shape[0] - 1), _ptr(qkv_out), _ptr(bg_out),
        _stream()), "gdn_prepare")


_GDN_CHUNKS = os.environ.get("TOKB200_GDN_SCAN", "tokens") == "chunks"


def gdn_scan(qkv: torch.Tensor, bg: torch.Tensor, groups: int, heads: int, dim: int, vdim: int, state: torch.Tensor,
             q_start, state_slot, o_out: torch.Tensor, longest: int = 1, chunks: Optional[bool] = None) -> None:
    """The recurrence S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q over every request's rows,
    head by head; `state` float32 [slots, n] holds the heads' matrices transposed and padded
    ([heads, vdim, gdn_padded_dim(dim)]) at the start of a slot; `o_out` float32 [T, heads * vdim].  `longest`: the
    most rows a request brings.  `chunks`: from 32 rows on, heads of 65 to 128 lanes run the chunk form of the rule
    (the same sums in another order; measured slower, so it is off unless asked for here or by TOKB200_GDN_SCAN=chunks)."""
    if chunks is None:
        chunks = _GDN_CHUNKS
    n = qkv.shape[0]
    if state.dtype != torch.float32 or o_out.dtype != torch.float32 or tuple(o_out.shape) != (n, heads * vdim) or \
            qkv.shape[1] != 2 * groups * dim + heads * vdim or heads * vdim * gdn_padded_dim(dim) > state.shape[1] or \
            tuple(bg.shape) != (n, 2 * heads + groups) or bg.dtype != torch.float32:
        raise ValueError("gdn_scan: sizes of the state or the outputs disagree")
    _check(_lib("delta_rule").tokb200_gdn_scan(
        _ptr(qkv), _ptr(bg), _i(groups), _i(heads), _i(dim), _i(vdim), _ptr(state), _ll(state.shape[1]),
        _ptr(q_start), _ptr(state_slot), _i(q_start.shape[0] - 1), _i(longest), _i(int(bool(chunks))), _ptr(o_out),
        _stream()), "gdn_scan")


def gdn_step_supported(dim: int, vdim: int) -> bool:
    """Whether a step of single tokens runs as one kernel (a block holds all of a head's columns)."""
    return bool(_lib("delta_rule").tokb200_gdn_step_supported(_i(dim), _i(vdim)))


def gdn_step(proj: torch.Tensor, qkv_at: int, b_at: int, a_at: int, g_at: int, groups: int, heads: int, dim: int,
             vdim: int, taps: int, conv_w, a_log, dt_bias, gain, scale: float, eps: float, state: torch.Tensor,
             conv_off: int, row_req, q_start, state_slot, out: torch.Tensor) -> None:
    """A step in which every request brings ONE token: what `gdn_prepare`, `gdn_scan` and `gdn_out_norm` do,
    in one kernel (a block a row and head), then the kept inputs move on.  `out` [T, heads * vdim]."""
    channels = 2 * groups * dim + heads * vdim
    n = proj.shape[0]
    if state.dtype != torch.float32 or state.dim() != 2 or tuple(out.shape) != (n, heads * vdim) or \
            conv_w.numel() != channels * taps or conv_off + (taps - 1) * channels > state.shape[1] or \
            gain.numel() != vdim or g_at + heads * vdim > proj.shape[1]:
        raise ValueError("gdn_step: sizes of the state, the taps, the gain or the output disagree")
    _check(_lib("delta_rule").tokb200_gdn_step(
        _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(qkv_at), _i(b_at), _i(a_at), _i(g_at), _i(groups), _i(heads),
        _i(dim), _i(vdim), _i(taps), _ptr(conv_w), _ptr(a_log), _ptr(dt_bias), _ptr(gain), _f(scale), _f(eps), _ptr(state),
        _ll(state.shape[1]), _i(conv_off), _ptr(row_req), _ptr(q_start), _ptr(state_slot), _i(n), _i(q_start.shape[0] - 1),
        _ptr(out), _i(_tag(out)), _stream()), "gdn_step")


def gdn_out_norm(o: torch.Tensor, gate: torch.Tensor, g_at: int, gain: torch.Tensor, scale: float, eps: float,
                 out: torch.Tensor, heads: int, vdim: int, row_req, gate_kind: str = "silu") -> None:
    """out[t, h] = o[t, h] / sqrt(mean(o[t, h]^2) + eps) * gain * scale * silu(gate[t, g_at + h vdim ..]), or the
    sigmoid of the gate (`gate_kind` "sigmoid")."""
    if gate_kind not in ("silu", "sigmoid"):
        raise ValueError("gdn_out_norm: the gate is silu or sigmoid")
    n = o.shape[0]
    if o.dtype != torch.float32 or tuple(o.shape) != (n, heads * vdim) or tuple(out.shape) != (n, heads * vdim) or \
            gain.numel() != vdim or g_at + heads * vdim > gate.shape[1]:
        raise ValueError("gdn_out_norm: o float32 [T, heads * vdim], a gain of vdim, the gate's columns inside its matrix")
    _check(_lib("delta_rule").tokb200_gdn_out_norm(
        _ptr(o), _sliced_ptr(gate), _i(_tag(gate)), _i(_ld(gate)), _i(g_at), _ptr(gain), _f(scale), _f(eps), _ptr(out),
        _i(_tag(out)), _i(n), _i(heads), _i(vdim), _ptr(row_req), _i(int(gate_kind == "sigmoid")), _stream()),
        "gdn_out_norm")


# ---- the delta rule with a decay a key channel ----
CDR_RUN = 4        # tokens of a run (csrc/channel_delta.cu)


def cdr_padded_dim(dim: int) -> int:
    """Rows of a head's state column as the recurrence keeps it; 0: a size it does not take."""
    return int(_lib("channel_delta").tokb200_cdr_padded_dim(_i(dim)))


def cdr_record(dim: int, vdim: int) -> int:
    """Floats of the record that `cdr_prepare` makes of one run and head."""
    return int(_lib("channel_delta").tokb200_cdr_record(_i(dim), _i(vdim)))


def cdr_records(n_rows: int, n_requests: int, heads: int, dim: int, vdim: int, device) -> torch.Tensor:
    """Room for a step's records: every request's portion is cut into runs of four rows."""
    return torch.empty((n_rows // CDR_RUN + n_requests, heads, cdr_record(dim, vdim)), dtype=torch.float32, device=device)


def cdr_prepare(proj: torch.Tensor, qkv_at: int, b_at: int, pre: torch.Tensor, groups: int, heads: int, dim: int,
                vdim: int, taps: int, conv_w, a_log, dt_bias, state: torch.Tensor, conv_off: int, q_start, state_slot,
                records: torch.Tensor) -> None:
    """Short convolution + silu of q, k, v (from `proj`'s columns qkv_at ..), unit vectors for q (times
    dim^-1/2) and k, beta = sigmoid(proj[b_at ..]) and the decays exp(-exp(a_log) softplus(pre + dt_bias)), one a head and
    key channel (`pre` float32, its first heads * dim columns), made into one record a run of four rows and
    head (`cdr_records`).  The kept inputs in `state` are read, not moved on (`short_conv_state` does that)."""
    channels, n = 2 * groups * dim + heads * vdim, proj.shape[0]
    if proj.dtype != torch.float32 or pre.dtype != torch.float32 or pre.shape[0] != n or pre.shape[1] < heads * dim or \
            state.dtype != torch.float32 or state.dim() != 2 or conv_w.numel() != channels * taps or \
            conv_off + (taps - 1) * channels > state.shape[1] or max(qkv_at + channels, b_at + heads) > proj.shape[1] or \
            a_log.numel() != heads or dt_bias.numel() != heads * dim or \
            tuple(records.shape[1:]) != (heads, cdr_record(dim, vdim)) or \
            records.shape[0] < n // CDR_RUN + q_start.shape[0] - 1:
        raise ValueError("cdr_prepare: sizes of the products, the state, the taps or the records disagree")
    _check(_lib("channel_delta").tokb200_cdr_prepare(
        _sliced_ptr(proj), _i(_ld(proj)), _i(qkv_at), _i(b_at), _sliced_ptr(pre), _i(_ld(pre)), _i(groups), _i(heads), _i(dim),
        _i(vdim), _i(taps), _ptr(conv_w), _ptr(a_log), _ptr(dt_bias), _ptr(state), _ll(state.shape[1]), _i(conv_off),
        _ptr(q_start), _ptr(state_slot), _i(n), _i(q_start.shape[0] - 1), _ptr(records), _stream()), "cdr_prepare")


def cdr_scan(records: torch.Tensor, heads: int, dim: int, vdim: int, state: torch.Tensor, q_start, state_slot,
             o_out: torch.Tensor) -> None:
    """The recurrence over every request's runs, head by head; `state` float32 [slots, n] holds the heads'
    matrices transposed and padded ([heads, vdim, cdr_padded_dim(dim)]) at the start of a slot; `o_out` float32
    [T, heads * vdim]."""
    if state.dtype != torch.float32 or o_out.dtype != torch.float32 or o_out.shape[1] != heads * vdim or \
            heads * vdim * cdr_padded_dim(dim) > state.shape[1] or tuple(records.shape[1:]) != (heads, cdr_record(dim, vdim)):
        raise ValueError("cdr_scan: sizes of the state, the records or the output disagree")
    _check(_lib("channel_delta").tokb200_cdr_scan(
        _ptr(records), _i(heads), _i(dim), _i(vdim), _ptr(state), _ll(state.shape[1]), _ptr(q_start), _ptr(state_slot),
        _i(q_start.shape[0] - 1), _ptr(o_out), _stream()), "cdr_scan")


def cdr_step(proj: torch.Tensor, qkv_at: int, b_at: int, low_at: int, ra: int, rg: int, w2, pre, groups: int, heads: int,
             dim: int, vdim: int, taps: int, conv_w, a_log, dt_bias, gain, eps: float, state: torch.Tensor, conv_off: int,
             row_req, state_slot, shift: bool, out: torch.Tensor) -> None:
    """A step in which every request brings ONE token: convolution, decay, recurrence, output norm and the sigmoid
    gate in one kernel.  `pre` float32 [T, heads * (dim + vdim)]: the pre-activations of the decay and of the gate;
    None: the kernel makes them from `proj`'s columns low_at .. + ra + rg and `w2` [heads * (dim + vdim), ra + rg].
    `shift`: the kept inputs move on here (every head has q and k of its own); else `short_conv_state` follows."""
    channels, n = 2 * groups * dim + heads * vdim, proj.shape[0]
    if proj.dtype != torch.float32 or state.dtype != torch.float32 or state.dim() != 2 or tuple(out.shape) != (n, heads * vdim) or \
            conv_w.numel() != channels * taps or conv_off + (taps - 1) * channels > state.shape[1] or gain.numel() != vdim or \
            (shift and heads != groups) or a_log.numel() != heads or dt_bias.numel() != heads * dim:
        raise ValueError("cdr_step: sizes of the state, the taps, the gain or the output disagree")
    if (pre is None and (tuple(w2.shape) != (heads * (dim + vdim), ra + rg) or w2.dtype != out.dtype or
                         low_at + ra + rg > proj.shape[1])) or \
            (pre is not None and (pre.dtype != torch.float32 or tuple(pre.shape) != (n, heads * (dim + vdim)))):
        raise ValueError("cdr_step: the second low-rank products or their weight have other sizes")
    _check(_lib("channel_delta").tokb200_cdr_step(
        _sliced_ptr(proj), _i(_ld(proj)), _i(qkv_at), _i(b_at), _i(low_at), _i(ra), _i(rg), _ptr(w2), _i(_tag(out)),
        _ptr(pre), _i(groups), _i(heads), _i(dim), _i(vdim), _i(taps), _ptr(conv_w), _ptr(a_log), _ptr(dt_bias), _ptr(gain),
        _f(eps), _ptr(state), _ll(state.shape[1]), _i(conv_off), _ptr(row_req), _ptr(state_slot), _i(n), _i(int(bool(shift))),
        _ptr(out), _i(_tag(out)), _stream()), "cdr_step")


def take_columns(proj: torch.Tensor, at: int, out: torch.Tensor) -> None:
    """out [T, n] (dense) = columns at .. + n of the float32 product `proj`."""
    n_rows, n = out.shape
    if proj.dtype != torch.float32 or proj.shape[0] != n_rows or at + n > proj.shape[1]:
        raise ValueError("take_columns: a float32 product that has the columns")
    _check(_lib("channel_delta").tokb200_take_columns(
        _sliced_ptr(proj), _i(_ld(proj)), _i(at), _i(n), _ptr(out), _i(_tag(out)), _i(n_rows), _stream()), "take_columns")


# ---- a norm without statistics and the stream's steps around it ----
def stream_update(x: torch.Tensor, y=None, base=None, carried=None, share=None, alpha=None, gain=None, bias=None,
                  beside=None, out=None, rows=None) -> None:
    """x <- (x or `base`, a float32 vector over the width) + y + share * carried, in place (each where given; x
    float32 [T, H]; y [T, H] or float32 partial sums [S, T, H]; `carried` [T, H] with one float32 a row in `share`,
    a column of a wider matrix).  With `out`: out = tanh(alpha x) * gain + bias of the new x, or x itself where `gain` is None; with
    `beside` (float32 [T, H]) out is [T, 2 H] and its second half is `beside`.  `rows` (int32): only those rows of x
    are read and x stays as it is."""
    hidden = x.shape[-1]
    n_rows = x.shape[0] if rows is None else rows.shape[0]
    if x.dtype != torch.float32 or (gain is not None and (out is None or gain.dtype != torch.float32 or bias.dtype != torch.float32 or
                                                          gain.numel() != hidden or bias.numel() != hidden)) or \
            (out is not None and tuple(out.shape) != (n_rows, hidden * (2 if beside is not None else 1))) or \
            (carried is not None and (tuple(carried.shape) != tuple(x.shape) or share.dtype != torch.float32 or
                                      share.numel() != n_rows)) or \
            (base is not None and (base.dtype != torch.float32 or base.numel() != hidden)) or \
            (beside is not None and (beside.dtype != torch.float32 or beside.shape != x.shape)):
        raise ValueError("stream_update: x is float32 [T, H]; vectors are float32 of H, matrices [T, H]")
    n_partials, stride = _partials(y, x) if y is not None else (1, 0)
    _check(_lib("dynamic_tanh").tokb200_stream_update(
        _ptr(x), _ptr(y), _i(_tag(y) if y is not None else F32), _i(n_partials), _ll(stride), _ptr(base), _ptr(carried),
        _i(_tag(carried) if carried is not None else F32), _sliced_ptr(share) if share is not None else _ptr(None),
        _i(share.stride(0) if share is not None else 0), _i(int(gain is not None)), _f(alpha if alpha is not None else 0.0), _ptr(gain), _ptr(bias),
        _ptr(beside), _ptr(out), _i(_tag(out) if out is not None else F32), _i(out.shape[1] if out is not None else 0),
        _ptr(rows), _i(n_rows), _i(hidden), _stream()), "stream_update")


# ---- queries, keys and values with unlike head sizes; routed experts ----
def qkv_rotate_store(proj: torch.Tensor, at: int, bias, inv_freq, rot_dims: int, pos, slot, row_req, q_out, k_pool,
                     v_pool, heads: int, kv_heads: int, dim: int, vdim: int, row: int, q_gain=None, k_gain=None,
                     eps: float = 0.0, temp=None, layout: str = "interleaved", head_norm_eps: Optional[float] = None,
                     magnitude: float = 1.0, values_are_keys: bool = False) -> None:
    """Bias, interleaved rotation of the first `rot_dims` lanes of every query and key head, and the
    cache write, from `proj`'s columns at .. (q, k, v); rows of `row` lanes a head, zero behind dim
    (queries, keys) and vdim (values).  `slot` None: no cache write.  `q_gain` / `k_gain` (float32, one a
    column of q / of k): the whole q (k) projection of a token is divided by its root mean square (`eps`
    inside the root) and multiplied by the gain first; `temp` (float32, one a query head) multiplies
    the head's queries.  `layout` "half": lane i of the rotated lanes pairs with lane i + rot_dims / 2 instead.
    `head_norm_eps` (a number): after the rotation every query and key head is divided by its own root mean
    square over its dim lanes, that eps inside the root.  `inv_freq` float64: the angle position * frequency is
    taken in 64-bit and brought into one turn before its sine and cosine (float32: the 32-bit product).  `magnitude` multiplies cosine and sine (1 with `head_norm_eps`).  `kv_heads` 0: `proj` holds queries only and nothing
    but `q_out` is written (`slot`, `k_pool`, `v_pool` None).  `values_are_keys`: `proj` has no v columns; a
    token's values are its keys as projected (bias added; no norm, no rotation), vdim = dim."""
    n = proj.shape[0]
    if values_are_keys and (vdim != dim or kv_heads == 0):
        raise ValueError("qkv_rotate_store: values that are the keys have the keys' lanes")
    if layout not in ("interleaved", "half"):
        raise ValueError("qkv_rotate_store: the rotated lanes pair interleaved or by halves")
    if kv_heads == 0 and (slot is not None or k_gain is not None):
        raise ValueError("qkv_rotate_store: a projection of queries alone writes no cache rows")
    if tuple(q_out.shape) != (n, heads * row) or \
            (kv_heads and (k_pool.dtype != q_out.dtype or v_pool.dtype != q_out.dtype)) or \
            at + heads * dim + kv_heads * (dim if values_are_keys else dim + vdim) > proj.shape[1]:
        raise ValueError("qkv_rotate_store: q_out is [T, heads * row] in the cache's type, the columns inside proj")
    for gain, size in ((q_gain, heads * dim), (k_gain, kv_heads * dim), (temp, heads)):
        if gain is not None and (gain.dtype != torch.float32 or gain.numel() != size):
            raise ValueError("qkv_rotate_store: gains are float32, one a column of q and of k; temperatures one a head")
    wide = inv_freq is not None and inv_freq.dtype == torch.float64      # frequencies in 64-bit: the angle is too
    _check(_lib("rotary_store").tokb200_qkv_rotate_store(
        _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(at), _ptr(bias), _ptr(None if wide else inv_freq),
        _ptr(inv_freq if wide else None), _i(rot_dims), _ptr(pos),
        _ptr(slot), _ptr(row_req), _ptr(q_out), _ptr(k_pool), _ptr(v_pool), _i(_tag(q_out)), _i(n), _i(heads),
        _i(kv_heads), _i(dim), _i(vdim), _i(row), _ptr(q_gain), _ptr(k_gain), _f(eps), _ptr(temp),
        _i(int(layout == "half")), _i(int(head_norm_eps is not None)), _f(head_norm_eps or 0.0), _f(magnitude),
        _i(int(values_are_keys)), _stream()), "qkv_rotate_store")


def attention_gate(out: torch.Tensor, proj: torch.Tensor, at: int, heads: int, vdim: int, row: int) -> None:
    """out[t, h, l] *= sigmoid(proj[t, at + h * vdim + l]) for l < vdim, in place; `out` is [T, heads * row]
    (the heads' outputs on rows of `row` lanes), the gate's pre-activations are columns at .. of `proj`."""
    n = out.shape[0]
    if tuple(out.shape) != (n, heads * row) or proj.shape[0] != n or at + heads * vdim > proj.shape[1] or row < vdim:
        raise ValueError("attention_gate: out is [T, heads * row], the gate's columns lie inside proj")
    _check(_lib("rotary_store").tokb200_attention_gate(
        _ptr(out), _i(_tag(out)), _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(at), _i(n), _i(heads), _i(vdim),
        _i(row), _stream()), "attention_gate")


MOE_SCORES = {"softmax_of_chosen": 0, "sigmoid": 1, "softmax": 2}
MOE_SHARED = {None: 0, "gated": 1, "one": 2}
MOE_ACTIVATIONS = dict(ACTIVATIONS, clamped_swish=len(ACTIVATIONS))


def moe_route(h: torch.Tensor, w: torch.Tensor, experts: int, top: int, shared, share: torch.Tensor,
              score: str = "softmax_of_chosen", correction: Optional[torch.Tensor] = None, groups: int = 1,
              keep: int = 1, scale: float = 1.0, identity: int = 0, group_worth: int = 2,
              renormalize: bool = False) -> None:
    """Router logits z = w h in 32-bit (`w` float32 [experts (+ 1), hidden]; `h` float32 or bfloat16), then
    every expert's share of the token, zero where it is not chosen.  `score` "softmax_of_chosen": the `top`
    largest logits, share = softmax over them.  "sigmoid": s = sigmoid(z); the choice is made on s +
    `correction` (float32, one an expert, or None) among the experts of the `keep` best of `groups` equal
    groups of neighbours (a group's worth: the sum of its `group_worth` largest choice scores, 1 or 2); share =
    s * `scale`, divided by the chosen scores' sum + 1e-20 where `renormalize` says so.  "softmax": the same with s
    the softmax over all router outputs.  `identity` (not with "softmax_of_chosen"): that many router rows behind the
    experts' stand for the token's input itself; they are chosen like experts (groups and correction run over both),
    and the sum of their shares is one more column of `share`, the last.
    `shared`: None / False (no shared expert), "gated" / True (share[t, experts] = sigmoid of one more router
    row), "one" (share[t, experts] = 1)."""
    n, hidden = h.shape
    shared = {True: "gated", False: None}.get(shared, shared)
    rows = experts + identity + int(shared == "gated")
    columns = experts + int(shared is not None) + int(identity > 0)
    if w.dtype != torch.float32 or tuple(w.shape) != (rows, hidden) or share.dtype != torch.float32 or \
            tuple(share.shape) != (n, columns):
        raise ValueError("moe_route: float32 router rows [experts (+ 1), hidden], shares float32 [T, experts (+ 1)]")
    if correction is not None and (correction.dtype != torch.float32 or correction.numel() != experts + identity):
        raise ValueError("moe_route: the correction is float32, one an expert")
    _check(_lib("moe").tokb200_moe_route(_ptr(h), _i(_tag(h)), _ptr(w), _i(hidden), _i(experts), _i(top),
                                         _i(MOE_SHARED[shared]), _ptr(share), _i(n), _i(MOE_SCORES[score]),
                                         _ptr(correction), _i(groups), _i(keep), _f(scale), _i(identity), _i(group_worth),
                                         _i(int(bool(renormalize))), _stream()), "moe_route")


def moe_gate(gu: torch.Tensor, share: torch.Tensor, out: torch.Tensor, experts: int, ff: int, shared: bool,
             activation: str = "silu", limit: float = 0.0, shared_limit: float = 0.0, alpha: float = 1.0,
             on_input: bool = False) -> None:
    """out[t, c] = act(gu[t, c]) * gu[t, I + c] * share[t, expert of lane c]: lanes 0 .. experts * ff
    are the routed experts' (ff each), the lanes behind the shared expert's.  `activation` is one of
    MOE_ACTIVATIONS; "clamped_swish": with g = min(gate, limit), u = clamp(up, -limit, limit), the lane is
    g * sigmoid(alpha g) * (u + 1) (`shared_limit` for the shared expert's lanes).  `on_input`: the share
    multiplies the expert's input instead, out[t, c] = act(share * gate) * (share * up)."""
    n, inner = out.shape
    if gu.shape[1] != 2 * inner or gu.dtype != out.dtype or share.shape[0] != n or share.shape[1] < experts + int(shared):
        raise ValueError("moe_gate: input [T, 2 I], output [T, I] of one type, shares [T, experts (+ 1) or more]")
    if activation not in MOE_ACTIVATIONS:
        raise ValueError(f"moe_gate: activation is one of {', '.join(MOE_ACTIVATIONS)}")
    _check(_lib("moe").tokb200_moe_gate(_ptr(gu), _ptr(share), _ptr(out), _i(_tag(gu)), _i(n), _i(inner), _i(experts),
                                        _i(ff), _i(int(shared)), _i(MOE_ACTIVATIONS[activation]), _f(limit),
                                        _f(shared_limit), _f(alpha), _i(int(on_input)), _i(share.shape[1]), _stream()),
           "moe_gate")


# ---- a short convolution across steps; a layer whose sublayers share one norm; learned positions ----
CONV_ACTIVATIONS = {None: 0, "silu": 1}


def short_conv(x: torch.Tensor, at: int, channels: int, w: torch.Tensor, bias, state, off: int, row_req, q_start,
               state_slot, out: torch.Tensor, activation=None, residual: bool = False, shift: bool = False) -> None:
    """out[t, c] = f(sum_j w[c, j] x[t - (taps - 1) + j, at + c] + bias[c]) (+ x[t, at + c] with `residual`)
    over the rows of each request; rows before a request's first row of the step are the taps - 1 inputs kept
    in `state` (float32 [slots, n], at `off` in the request's slot, [taps - 1, channels]).  `w` float32
    [channels, taps]; `out` [T, channels] dense."""
    n = x.shape[0]
    taps = w.shape[1]
    if w.dtype != torch.float32 or tuple(w.shape) != (channels, taps) or tuple(out.shape) != (n, channels) or \
            at + channels > x.shape[1] or (bias is not None and (bias.dtype != torch.float32 or bias.numel() != channels)) or \
            (taps > 1 and (state is None or state.dtype != torch.float32 or state.dim() != 2)):
        raise ValueError("short_conv: taps float32 [channels, taps], out [T, channels], a float32 state [slots, n]")
    _check(_lib("short_conv").tokb200_short_conv(
        _sliced_ptr(x), _i(_tag(x)), _i(_ld(x)), _i(at), _i(channels), _i(taps), _ptr(w), _ptr(bias),
        _ptr(state if taps > 1 else None), _ll(state.shape[1] if taps > 1 else 0), _i(off), _ptr(row_req), _ptr(q_start),
        _ptr(state_slot), _i(CONV_ACTIVATIONS[activation]), _i(int(residual)), _ptr(out), _i(_tag(out)), _i(n),
        _i(int(shift)), _stream()), "short_conv")


def short_conv_state(x: torch.Tensor, at: int, channels: int, taps: int, state: torch.Tensor, off: int, q_start,
                     state_slot) -> None:
    """The kept inputs of `short_conv` move on by the step's rows; launch it behind the convolution."""
    if taps <= 1:
        return
    if state.dtype != torch.float32 or state.dim() != 2 or at + channels > x.shape[1]:
        raise ValueError("short_conv_state: a float32 state [slots, n], the channels inside x")
    _check(_lib("short_conv").tokb200_short_conv_state(
        _sliced_ptr(x), _i(_tag(x)), _i(_ld(x)), _i(at), _i(channels), _i(taps), _ptr(state), _ll(state.shape[1]),
        _i(off), _ptr(q_start), _ptr(state_slot), _i(q_start.shape[0] - 1), _stream()), "short_conv_state")


def scaled_add_norm(x: torch.Tensor, terms, gain: Optional[torch.Tensor] = None, eps: float = 0.0,
                    out: Optional[torch.Tensor] = None) -> None:
    """x += sum of vector * term over one or two `terms` ((tensor [T, H] or float32 partial sums [S, T, H],
    float32 vector [H])), in place (x float32); with `gain`, also out = x / sqrt(mean(x^2) + eps) * gain of
    the new x."""
    n_rows, hidden = x.shape
    if x.dtype != torch.float32 or not 1 <= len(terms) <= 2 or \
            any(v.dtype != torch.float32 or v.numel() != hidden for _, v in terms):
        raise ValueError("scaled_add_norm: x float32 [T, H], one or two terms with float32 vectors of H")
    if gain is not None and (out is None or tuple(out.shape) != (n_rows, hidden) or gain.numel() != hidden):
        raise ValueError("scaled_add_norm: the norm behind the add needs a gain of H and out [T, H]")
    args = []
    for term in list(terms) + [None] * (2 - len(terms)):
        if term is None:
            args += [_ptr(None), _i(F32), _i(1), _ll(0), _ptr(None)]
        else:
            y, v = term
            n_partials, stride = _partials(y, x)
            args += [_ptr(y), _i(_tag(y)), _i(n_partials), _ll(stride), _ptr(v)]
    _check(_lib("short_conv").tokb200_scaled_add_norm(
        _ptr(x), *args, _ptr(gain), _f(eps), _ptr(out), _i(_tag(out) if out is not None else F32), _i(n_rows),
        _i(hidden), _stream()), "scaled_add_norm")


def embed_positions(ids: torch.Tensor, pos: torch.Tensor, row_req: torch.Tensor, table: torch.Tensor,
                    positions: torch.Tensor, out: torch.Tensor, scale: float = 1.0) -> None:
    """out[t] = table[ids[t]] * scale + positions[pos[t]], float32."""
    n, hidden = out.shape
    if table.dtype != positions.dtype or table.shape[1] != hidden or positions.shape[1] != hidden:
        raise ValueError("embed_positions: both tables have rows of the stream's width and one type")
    _check(_lib("short_conv").tokb200_embed_positions(
        _ptr(ids), _ptr(pos), _ptr(row_req), _ptr(table), _ptr(positions), _i(_tag(table)), _ptr(out), _i(n), _i(hidden),
        _i(table.shape[0]), _i(positions.shape[0]), _f(scale), _stream()), "embed_positions")


# ---- the selective state-space recurrence (scalar decay a head) ----
MAMBA2_MAX_STATE = 256


_M2_SEGMENTS = int(os.environ.get("TOKB200_M2_SEGMENTS", "0"))     # > 0: that many segments a request, whatever the step
MAMBA2_MAX_SEGMENTS = 16


def mamba2_segments(n_rows: int, n_requests: int, heads: int, vdim: int) -> int:
    """Into how many segments that run side by side `mamba2_scan` cuts a request's rows: as many as give every
    multiprocessor a few blocks (a block is 32 columns of a head and request), none shorter than 64 rows on
    average; 1 for steps whose requests fill the device by themselves and for decoding steps.  It depends on
    the step's shape alone, so a captured step replays with the same launches."""
    if _M2_SEGMENTS > 0:
        return min(_M2_SEGMENTS, MAMBA2_MAX_SEGMENTS)
    blocks = -(-vdim // 32) * heads * max(1, n_requests)
    return max(1, min(592 // blocks, n_rows // (64 * max(1, n_requests)), MAMBA2_MAX_SEGMENTS))


def mamba2_scan(xbc: torch.Tensor, proj: torch.Tensor, dt_at: int, dt_bias, a_log, skip, heads: int, groups: int,
                vdim: int, n_state: int, state: torch.Tensor, q_start, state_slot, y: torch.Tensor,
                segments: Optional[int] = None) -> None:
    """Per head and token: dt = softplus(proj[dt_at + head] + dt_bias); S <- exp(-exp(a_log) dt) S + dt B x^T;
    y = S^T C + skip x, over every request's rows.  `xbc` float32 [T, heads * vdim + 2 groups * n_state] (x, B,
    C); `state` float32 [slots, n] with a slot's matrices [heads, vdim, n_state] at its start; `y` float32
    [T, heads * vdim].  `segments` > 1: every request's rows of the step are cut into that many equal segments
    that run side by side (the recurrence is linear in S: a segment's end is the product of its decays times
    its start plus its end from a zero start), two launches; None: `mamba2_segments` chooses."""
    n = xbc.shape[0]
    if xbc.dtype != torch.float32 or y.dtype != torch.float32 or tuple(y.shape) != (n, heads * vdim) or \
            xbc.shape[1] != heads * vdim + 2 * groups * n_state or state.dtype != torch.float32 or state.dim() != 2 or \
            dt_at + heads > proj.shape[1] or any(v.dtype != torch.float32 or v.numel() != heads for v in (dt_bias, a_log, skip)):
        raise ValueError("mamba2_scan: sizes of the inputs, the state or the output disagree")
    n_requests = q_start.shape[0] - 1
    if segments is None:
        segments = mamba2_segments(n, n_requests, heads, vdim)
    if not 1 <= segments <= MAMBA2_MAX_SEGMENTS:
        raise ValueError(f"mamba2_scan: 1 to {MAMBA2_MAX_SEGMENTS} segments")
    # the segments' ends (as the slot's matrices) and the products of their decays
    scratch = torch.empty(n_requests * segments * heads * (vdim * n_state + 1), dtype=torch.float32,
                          device=xbc.device) if segments > 1 else None
    _check(_lib("mamba2").tokb200_mamba2_scan(
        _ptr(xbc), _i(xbc.shape[1]), _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(dt_at), _ptr(dt_bias), _ptr(a_log),
        _ptr(skip), _i(heads), _i(groups), _i(vdim), _i(n_state), _ptr(state), _ll(state.shape[1]), _ptr(q_start),
        _ptr(state_slot), _i(n_requests), _ptr(y), _ptr(scratch), _i(segments), _stream()), "mamba2_scan")
    if segments > 1:
        counter.launches += 1


def mamba2_out_norm(y: torch.Tensor, proj: torch.Tensor, z_at: int, gain: torch.Tensor, eps: float, parts: int,
                    row_req, out: torch.Tensor) -> None:
    """out = (y * silu(proj[:, z_at ..])) divided by its root mean square inside each of `parts` equal parts of
    the row (eps inside the root), times `gain` (float32, one a lane)."""
    n, inner = y.shape
    if y.dtype != torch.float32 or tuple(out.shape) != (n, inner) or gain.dtype != torch.float32 or gain.numel() != inner or \
            z_at + inner > proj.shape[1] or inner % parts:
        raise ValueError("mamba2_out_norm: y float32 [T, inner], a gain of inner, the gate's columns inside proj")
    _check(_lib("mamba2").tokb200_mamba2_out_norm(
        _ptr(y), _sliced_ptr(proj), _i(_tag(proj)), _i(_ld(proj)), _i(z_at), _ptr(gain), _f(eps), _i(inner), _i(parts),
        _ptr(row_req), _ptr(out), _i(_tag(out)), _i(n), _stream()), "mamba2_out_norm")


# ---- several residual streams ----
STREAMS_MAX = 8


def streams_step(x: torch.Tensor, streams: int, y=None, mix=None, share=None, read=None, gain=None, eps: float = 0.0,
                 out: Optional[torch.Tensor] = None, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x float32 [T, streams, H], or [T, H] where all streams are still equal.  With `y` ([T, H] or float32 partial sums
    [S, T, H]): x_t <- sum_s mix[s, t] x_s + share[t] y, in place (a new tensor where the streams were equal); returns
    the streams.  With `out` [T, H]: out = u, or u / sqrt(mean(u^2) + eps) * gain, u = sum_s read[s] x_s of the new
    streams (`read` None: their sum).  `rows` (int32): only those rows are read, `out` is dense, x stays as it is.
    mix [streams, streams] (from the row to the column), share and read [streams], gain [H]: float32."""
    equal, hidden = x.dim() == 2, x.shape[-1]
    n_rows = x.shape[0] if rows is None else rows.shape[0]
    if x.dtype != torch.float32 or (not equal and (x.dim() != 3 or x.shape[1] != streams)) or not 1 <= streams <= STREAMS_MAX:
        raise ValueError(f"streams_step: float32 [T, H] or [T, streams, H], 1 to {STREAMS_MAX} streams")
    for v, size in ((mix, streams * streams), (share, streams), (read, streams), (gain, hidden)):
        if v is not None and (v.dtype != torch.float32 or v.numel() != size):
            raise ValueError("streams_step: the weights are float32, one a stream (or pair of streams), the gain one a lane")
    if (y is not None and (mix is None or share is None)) or (out is not None and tuple(out.shape) != (n_rows, hidden)) or \
            (out is None and (gain is not None or y is None)):
        raise ValueError("streams_step: an output with its weights, a norm with its result [T, H]")
    flat = x if equal else x[:, 0]
    n_partials, stride = _partials(y, flat) if y is not None else (1, 0)
    x_out = None
    if y is not None and rows is None:
        x_out = torch.empty((x.shape[0], streams, hidden), dtype=torch.float32, device=x.device) if equal else x
    _check(_lib("streams").tokb200_streams_step(
        _ptr(x), _i(int(equal)), _ptr(x_out), _i(streams), _ptr(y), _i(_tag(y) if y is not None else F32), _i(n_partials),
        _ll(stride), _ptr(mix), _ptr(share), _ptr(read), _ptr(gain), _f(eps), _ptr(out),
        _i(_tag(out) if out is not None else F32), _ptr(rows), _i(n_rows), _i(hidden), _stream()), "streams_step")
    return x if x_out is None else x_out


# ---- attention over a latent: queries straight from the mixer's input, gated values ----
def latent_rotate_store(proj: torch.Tensor, c_at: int, q_at: int, heads: int, kv_rank: int, rot_dim: int, rot_dims: int,
                        row: int, c_gain, eps: float, inv_freq, pos, row_req, slot, q_out, pool) -> None:
    """From a float32 product's rows: the normed latent and the rotated positional key part into the token's cache row
    (`pool` [slots, 1, row]), and every head's query (columns q_at .., `row` a head) with its positional lanes rotated
    into `q_out` [T, heads * row].  `inv_freq` float64; `slot` None: no cache write."""
    n = proj.shape[0]
    if proj.dtype != torch.float32 or tuple(q_out.shape) != (n, heads * row) or pool.dtype != q_out.dtype or \
            pool.shape[-1] * pool.shape[-2] != row or q_at + heads * row > proj.shape[1] or \
            (inv_freq is not None and inv_freq.dtype != torch.float64):
        raise ValueError("latent_rotate_store: a float32 product, queries and pool of `row` lanes in one type, 64-bit frequencies")
    _check(_lib("latent").tokb200_latent_rotate_store(
        _sliced_ptr(proj), _i(_ld(proj)), _i(c_at), _i(q_at), _i(heads), _i(kv_rank), _i(rot_dim), _i(rot_dims), _i(row),
        _ptr(c_gain), _f(eps), _ptr(inv_freq), _ptr(pos), _ptr(row_req), _ptr(slot), _ptr(q_out), _ptr(pool), _i(_tag(pool)),
        _i(n), _stream()), "latent_rotate_store")


def latent_values(mixed: torch.Tensor, w: torch.Tensor, gate: torch.Tensor, g_at: int, heads: int, vdim: int, row: int,
                  out: torch.Tensor) -> None:
    """out[t, h] = (w[h] mixed[t, h]) * sigmoid(gate[t, g_at + h vdim ..]); `mixed` [T, heads * row], `out` [T, heads *
    vdim], `gate` a float32 product; w [heads, vdim, row] in bfloat16 (row in whole 16s), [heads, row, vdim] in float32."""
    n = mixed.shape[0]
    shape = (heads, vdim, row) if mixed.dtype == torch.bfloat16 else (heads, row, vdim)
    if tuple(mixed.shape) != (n, heads * row) or tuple(out.shape) != (n, heads * vdim) or tuple(w.shape) != shape or \
            w.dtype != mixed.dtype or out.dtype != mixed.dtype or gate.dtype != torch.float32 or gate.shape[0] != n or \
            g_at + heads * vdim > gate.shape[1]:
        raise ValueError("latent_values: sizes or types of the latents, the weights, the gate or the output disagree")
    _check(_lib("latent").tokb200_latent_values(
        _ptr(mixed), _ptr(w), _sliced_ptr(gate), _i(_ld(gate)), _i(g_at), _i(heads), _i(vdim), _i(row), _ptr(out),
        _i(_tag(out)), _i(n), _stream()), "latent_values")


# ---- the matrix memory with exponential gates ----
MLSTM_MAX_DIM = 256


def mlstm_gates(proj: torch.Tensor, i_at: int, f_at: int, i_bias, f_bias, cap: float, heads: int, state: torch.Tensor,
                m_off: int, q_start, state_slot, gates: torch.Tensor, start: Optional[torch.Tensor] = None) -> None:
    """The running maximum of every request's rows (`state` [slots, n]: it starts from and ends in the heads' numbers at
    m_off), and `gates` float32 [3, heads, >= T]: what a token's matrix is kept by, what its write is weighed by, and
    exp(-maximum).  With `start` (float32 [requests, heads], receives the maxima in front of the rows) `gates` holds the
    logarithms of the forget and input gates and the maxima themselves, as `mlstm_chunks` wants them."""
    if proj.dtype != torch.float32 or gates.dtype != torch.float32 or gates.shape[:2] != (3, heads) or \
            state.dtype != torch.float32 or state.dim() != 2 or \
            any(v.dtype != torch.float32 or v.numel() != heads for v in (i_bias, f_bias)):
        raise ValueError("mlstm_gates: a float32 product, biases one a head, gates [3, heads, T]")
    _check(_lib("mlstm").tokb200_mlstm_gates(
        _sliced_ptr(proj), _i(_ld(proj)), _i(i_at), _i(f_at), _ptr(i_bias), _ptr(f_bias), _f(cap), _i(heads), _ptr(state),
        _ll(state.shape[1]), _i(m_off), _ptr(q_start), _ptr(state_slot), _i(q_start.shape[0] - 1), _i(proj.shape[0]),
        _ptr(gates[0]), _ptr(gates[1]), _ptr(gates[2]), _ll(gates.shape[2]), _ptr(start), _stream()), "mlstm_gates")


def mlstm_chunks_supported(dim: int, vdim: int) -> bool:
    """Whether the form in chunks takes heads of these sizes."""
    return bool(_lib("mlstm_chunks").tokb200_mlstm_chunks_supported(_i(dim), _i(vdim)))


def mlstm_chunks(proj: torch.Tensor, q_at: int, k_at: int, v_at: int, g_at: int, heads: int, dim: int, vdim: int,
                 gates: torch.Tensor, start: torch.Tensor, gain, eps: float, state: torch.Tensor, q_start, state_slot,
                 out: torch.Tensor) -> None:
    """What `mlstm_scan` and `mlstm_out_norm` do, in chunks of 64 tokens on tensor cores (csrc/mlstm_chunks.cu), q, k and v
    as bfloat16 operands; `gates` and `start` from `mlstm_gates`.  `out` bfloat16 [T, heads * vdim]."""
    n, n_requests = proj.shape[0], q_start.shape[0] - 1
    if proj.dtype != torch.float32 or out.dtype != torch.bfloat16 or tuple(out.shape) != (n, heads * vdim) or \
            gates.dtype != torch.float32 or gates.shape[:2] != (3, heads) or gates.shape[2] < n or gain.numel() != heads * vdim or \
            start.dtype != torch.float32 or start.numel() != n_requests * heads or state.dtype != torch.float32 or \
            state.dim() != 2 or heads * (vdim + 1) * dim > state.shape[1]:
        raise ValueError("mlstm_chunks: sizes of the product, the gates, the state or the output disagree")
    places = n // 64 + n_requests
    sums = torch.empty(places * heads * (vdim + 1) * dim, dtype=torch.float32, device=proj.device)
    decay = torch.empty(places * heads, dtype=torch.float32, device=proj.device)
    _check(_lib("mlstm_chunks").tokb200_mlstm_chunks(
        _sliced_ptr(proj), _i(_ld(proj)), _i(q_at), _i(k_at), _i(v_at), _i(g_at), _i(heads), _i(dim), _i(vdim), _f(dim ** -0.5),
        _ptr(gates[0]), _ptr(gates[1]), _ptr(gates[2]), _ll(gates.shape[2]), _ptr(start), _ptr(q_start), _ptr(state_slot),
        _i(n_requests), _i(n), _ptr(state), _ll(state.shape[1]), _ptr(sums), _ptr(decay), _ptr(gain), _f(eps), _ptr(out),
        _stream()), "mlstm_chunks")
    counter.launches += 2


def mlstm_scan(proj: torch.Tensor, q_at: int, k_at: int, v_at: int, heads: int, dim: int, vdim: int, gates: torch.Tensor,
               state: torch.Tensor, q_start, state_slot, y: torch.Tensor, yn: torch.Tensor,
               segments: Optional[int] = None) -> None:
    """S <- keep S + add k v^T, n <- keep n + add k; y [T, heads * vdim] = S^T q dim^(-1/2), yn [T, heads] = n . q
    dim^(-1/2), over every request's rows; a slot of `state` starts with [heads, vdim + 1, dim] (n behind the columns).
    `segments` as for `mamba2_scan`."""
    n = proj.shape[0]
    if proj.dtype != torch.float32 or y.dtype != torch.float32 or tuple(y.shape) != (n, heads * vdim) or \
            tuple(yn.shape) != (n, heads) or yn.dtype != torch.float32 or gates.shape[:2] != (3, heads) or gates.shape[2] < n or \
            state.dtype != torch.float32 or state.dim() != 2 or heads * (vdim + 1) * dim > state.shape[1]:
        raise ValueError("mlstm_scan: sizes of the product, the gates, the state or the outputs disagree")
    n_requests = q_start.shape[0] - 1
    if segments is None:
        segments = mamba2_segments(n, n_requests, heads, vdim)
    if not 1 <= segments <= MAMBA2_MAX_SEGMENTS:
        raise ValueError(f"mlstm_scan: 1 to {MAMBA2_MAX_SEGMENTS} segments")
    scratch = torch.empty(n_requests * segments * heads * ((vdim + 1) * dim + 1), dtype=torch.float32,
                          device=proj.device) if segments > 1 else None
    _check(_lib("mlstm").tokb200_mlstm_scan(
        _sliced_ptr(proj), _i(_ld(proj)), _i(q_at), _i(k_at), _i(v_at), _i(heads), _i(dim), _i(vdim), _f(dim ** -0.5),
        _ptr(gates[0]), _ptr(gates[1]), _ll(gates.shape[2]), _ptr(state), _ll(state.shape[1]), _ptr(q_start), _ptr(state_slot),
        _i(n_requests), _ptr(y), _ptr(yn), _ptr(scratch), _i(segments), _stream()), "mlstm_scan")
    if segments > 1:
        counter.launches += 1


def mlstm_out_norm(y: torch.Tensor, yn: torch.Tensor, gates: torch.Tensor, proj: torch.Tensor, g_at: int, gain, eps: float,
                   heads: int, vdim: int, row_req, out: torch.Tensor) -> None:
    """o = y / (max(|yn|, exp(-maximum)) + 1e-6), divided by its root mean square over vdim, times `gain` (one a lane of
    all heads) and sigmoid(proj[:, g_at ..])."""
    n = y.shape[0]
    if tuple(out.shape) != (n, heads * vdim) or gain.numel() != heads * vdim or g_at + heads * vdim > proj.shape[1] or \
            proj.dtype != torch.float32 or gates.shape[2] < n:
        raise ValueError("mlstm_out_norm: sizes of the gain, the gate or the output disagree")
    _check(_lib("mlstm").tokb200_mlstm_out_norm(
        _ptr(y), _ptr(yn), _ptr(gates[2]), _ll(gates.shape[2]), _sliced_ptr(proj), _i(_ld(proj)), _i(g_at), _ptr(gain), _f(eps),
        _i(heads), _i(vdim), _ptr(row_req), _ptr(out), _i(_tag(out)), _i(n), _stream()), "mlstm_out_norm")


def mlstm_step(proj: torch.Tensor, q_at: int, k_at: int, v_at: int, g_at: int, i_at: int, f_at: int, i_bias, f_bias,
               cap: float, heads: int, dim: int, vdim: int, gain, eps: float, state: torch.Tensor, m_off: int, row_req,
               state_slot, out: torch.Tensor) -> None:
    """A step in which every request brings ONE token: gates, recurrence, norm and gate in one kernel, a block a (row,
    head)."""
    n = proj.shape[0]
    if proj.dtype != torch.float32 or tuple(out.shape) != (n, heads * vdim) or gain.numel() != heads * vdim or \
            state.dtype != torch.float32 or state.dim() != 2 or m_off < heads * (vdim + 1) * dim:
        raise ValueError("mlstm_step: sizes of the product, the state, the gain or the output disagree")
    _check(_lib("mlstm").tokb200_mlstm_step(
        _sliced_ptr(proj), _i(_ld(proj)), _i(q_at), _i(k_at), _i(v_at), _i(g_at), _i(i_at), _i(f_at), _ptr(i_bias), _ptr(f_bias),
        _f(cap), _i(heads), _i(dim), _i(vdim), _f(dim ** -0.5), _ptr(gain), _f(eps), _ptr(state), _ll(state.shape[1]), _i(m_off),
        _ptr(row_req), _ptr(state_slot), _i(n), _ptr(out), _i(_tag(out)), _stream()), "mlstm_step")


# ---- read-only streams in the decoding kernels' access patterns (bench.py --stream-probe) ----
STREAM_PATTERNS = {"coalesced": 0, "fragment": 1, "fragment_wide": 2}


def stream_probe_loads(w: torch.Tensor, pattern: str, in_flight: int, blocks: int, sink: torch.Tensor) -> None:
    """Read the bfloat16 matrix `w` [N, K] once with plain loads in one of STREAM_PATTERNS,
    `in_flight` (2, 4 or 8) steps of loads a thread, from `blocks` blocks of 256 threads."""
    N, K = w.shape
    _check(_lib("stream_probe").tokb200_stream_probe_loads(
        _ptr(w), _i(N), _i(K), _i(STREAM_PATTERNS[pattern]), _i(in_flight), _i(blocks), _ptr(sink), _stream()),
        "stream_probe_loads")


def stream_probe_bulk(w: torch.Tensor, piece_bytes: int, rows_per_stage: int, stages: int, blocks: int,
                      sink: torch.Tensor) -> None:
    """Read `w` once through a ring of shared-memory stages filled by bulk copies of `piece_bytes`
    of a row each (a stage: `rows_per_stage` pieces), one producer and one consumer warp a block."""
    N, K = w.shape
    _check(_lib("stream_probe").tokb200_stream_probe_bulk(
        _ptr(w), _i(N), _i(K), _i(piece_bytes), _i(rows_per_stage), _i(stages), _i(blocks), _ptr(sink), _stream()),
        "stream_probe_bulk")


def stream_probe_async_ring(w: torch.Tensor, depth: int, blocks: int, sink: torch.Tensor) -> None:
    """Read `w` once in the fragment pattern through rings of `depth` (4, 6 or 8) shared-memory
    stages a warp, filled by 16-byte asynchronous copies."""
    N, K = w.shape
    _check(_lib("stream_probe").tokb200_stream_probe_async_ring(
        _ptr(w), _i(N), _i(K), _i(depth), _i(blocks), _ptr(sink), _stream()), "stream_probe_async_ring")
