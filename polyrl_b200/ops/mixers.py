"""Sequence-mixer ops over packed spans: sm_100a kernels on CUDA tensors (bf16 or fp32), plain PyTorch on CPU tensors.

A ``SpanBatch`` describes one engine step: span ``s`` is the tokens ``[cu[s], cu[s + 1])`` of one sequence whose first
``start[s]`` tokens were processed earlier.  A decoded token is a span of one.  Recurrent state lives in pools indexed by
``slot``, keys in a paged pool indexed by ``kv_slot`` / ``table``; a span with ``start == 0`` begins from the zero state.
Spans are ordered: the ``n_long`` spans of several tokens first, then the single tokens.
"""
from __future__ import annotations

import math
from contextlib import contextmanager, nullcontext
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from .reference import split_gate_up

PAGE = 16


@dataclass
class SpanBatch:
    cu: torch.Tensor                    # [n + 1] int32
    start: torch.Tensor                 # [n] int32
    slot: torch.Tensor                  # [n] int64 state slot
    pos: torch.Tensor                   # [T] int64
    kv_slot: torch.Tensor               # [T] int64 flat cache row (page * PAGE + offset)
    kv_len: torch.Tensor                # [T] int32 keys a token sees, its own included (0: idle row)
    table: torch.Tensor                 # [n, width] int32 page numbers
    seq_of: torch.Tensor | None = None  # [T] int32 span of a token; None: every span is one token
    n_long: int = 0
    t_long: int = 0
    max_long: int = 0                   # longest span
    max_len: int = 0                    # bound on kv_len
    # keys of the long spans, per (window, kept first tokens) — (0, 0): all of them: (flat cache rows [Tk] int64, cu_k [n_long + 1]
    # int32), kept first tokens ahead of the window's; None: no span has earlier tokens
    gather: dict | None = None

    @property
    def spans(self) -> int:
        return self.start.numel()

    @property
    def tokens(self) -> int:
        return self.pos.numel()


def _C():
    from . import ext

    return ext()


_COUNTERS: dict = {}
_RETIRED: list = []     # outgrown counters stay alive: captured graphs hold their address


def _counter(device: torch.device, n: int, use: str = "scan") -> torch.Tensor:
    """Zeroed arrival counters of the recurrence and routing kernels (each launch leaves them zero again), one set per ``use``: the two may run
    at the same time; the last element is an error flag."""
    key = (device.type, device.index, use)
    if key not in _COUNTERS or _COUNTERS[key].numel() <= n:
        _RETIRED.append(_COUNTERS.get(key))
        _COUNTERS[key] = torch.zeros(max(n, 1 << 17) + 1, device=device, dtype=torch.int32)
    return _COUNTERS[key]


def check_errors(device: torch.device) -> None:
    """Raise if a bounded wait inside a kernel ran out (reads one flag back: call it where the host synchronises anyway)."""
    c = _COUNTERS.get((device.type, device.index, "scan"))
    if c is not None and int(c[-1]):
        raise RuntimeError("a wait inside a chunked recurrence kernel timed out")


_SIDE: dict = {}


@contextmanager
def beside(like: torch.Tensor, b: SpanBatch | None):
    """Two chains of small kernels next to each other in steps of single tokens:  ``with beside(x, b) as side: with side(): first()``; ``second()``.
    Elsewhere they run one after the other.  What the side stream allocates is reused only by its own later work, which waits for the kernel
    that consumed it; what it reads has to stay referenced until the outer block ends."""
    if b is None or not like.is_cuda or b.seq_of is not None:
        yield nullcontext
        return
    main = torch.cuda.current_stream(like.device)
    depth = next((d for (i, d), s in _SIDE.items() if i == like.device.index and s == main), 0) + 1
    if (like.device.index, depth) not in _SIDE:
        _SIDE[like.device.index, depth] = torch.cuda.Stream(device=like.device)
    other = _SIDE[like.device.index, depth]
    other.wait_stream(main)
    yield lambda: torch.cuda.stream(other)
    main.wait_stream(other)


# --------------------------------------------------------------------------------------------
# rows
# --------------------------------------------------------------------------------------------
def _rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def embed(ids: torch.Tensor, w: torch.Tensor, w_norm: torch.Tensor | None = None, eps: float = 0.0) -> tuple[torch.Tensor, torch.Tensor]:
    """(fp32 residual stream, the same in the activation dtype — one tensor when that is fp32); with ``w_norm`` the second is
    rms(x) * w_norm."""
    if w.is_cuda:
        return tuple(_C().mix_embed(ids, w, w_norm, eps))
    x = F.embedding(ids, w).float()
    if w_norm is not None:
        return x, (_rms(x, eps) * w_norm).to(w.dtype)
    return x, (x if w.dtype == torch.float32 else x.to(w.dtype))


def norm_add_(y: torch.Tensor, x: torch.Tensor, w: torch.Tensor, eps: float, w_next: torch.Tensor | None = None) -> torch.Tensor:
    """x += rms(y) * w (fp32, in place); returns x in y's dtype, or rms(x) * w_next in y's dtype."""
    if y.is_cuda:
        return _C().mix_norm_add_(y, x, w, eps, w_next)
    x.add_(_rms(y.float(), eps) * w)
    if w_next is not None:
        return (_rms(x, eps) * w_next).to(y.dtype)
    return x if y.dtype == torch.float32 else x.to(y.dtype)


def _norm(x: torch.Tensor, eps: float, center: bool) -> torch.Tensor:
    return _rms(x - x.mean(-1, keepdim=True) if center else x, eps)


def rms(x: torch.Tensor, w: torch.Tensor, eps: float, dtype: torch.dtype, center: bool = False) -> torch.Tensor:
    """rms(x) * w of fp32 rows in ``dtype``; ``center``: of x minus its mean (layer norm)."""
    if x.is_cuda:
        return _C().mix_rms(x.contiguous(), w, eps, dtype == torch.bfloat16, center)
    return (_norm(x, eps, center) * w).to(dtype)


SIGMOID_LAST, SILU_FIRST, SILU_LAST = 0, 1, 2


def gated_norm(y: torch.Tensor, z: torch.Tensor, w: torch.Tensor, groups: int, eps: float, gate: int, out: torch.Tensor | None = None) -> torch.Tensor:
    """Group RMS norm with a gate: rms(y) * w * sigmoid(z), rms(y * silu(z)) * w or rms(y) * w * silu(z), to ``out`` (rows of any pitch) when given."""
    if y.is_cuda:
        return _C().mix_gated_norm(y, z, w, groups, eps, gate, out)
    yf, zf = y.float(), z.float()
    if gate == SILU_FIRST:
        yf = yf * F.silu(zf)
    n = _rms(yf.reshape(y.shape[0], groups, -1), eps).reshape(y.shape) * w
    n = (n if gate == SILU_FIRST else n * (torch.sigmoid(zf) if gate == SIGMOID_LAST else F.silu(zf))).to(y.dtype)
    return n if out is None else out.copy_(n)


def linear_f32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """x @ w.T with the fp32 accumulator as the result (gates and step sizes of a recurrence)."""
    if x.is_cuda and x.dtype == torch.bfloat16:
        return torch.mm(x, w.t(), out_dtype=torch.float32)
    return F.linear(x.float(), w.float())


def linear_gelu(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """gelu_tanh(x @ w.T); fused into the GEMM epilogue for bf16 rows."""
    if x.is_cuda:
        if x.dtype == torch.bfloat16 and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0:
            return _C().gemm_gelu(x, w)
        y = F.linear(x, w)
        _C().mix_gelu_(y)
        return y
    return F.gelu(F.linear(x, w.to(x.dtype)), approximate="tanh")


def linear_silu(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """silu(x @ w.T); fused into the GEMM epilogue for bf16 rows."""
    if x.is_cuda:
        if x.dtype == torch.bfloat16 and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0:
            return _C().gemm_silu(x, w)
        y = F.linear(x, w)
        _C().mix_silu_(y)
        return y
    return F.silu(F.linear(x, w.to(x.dtype)))


def linear_clamped_glu(x: torch.Tensor, wgu: torch.Tensor, limit: float, alpha: float) -> torch.Tensor:
    """g sigmoid(alpha g) (u + 1) with g = min(gate, limit), u = clamp(up, -limit, limit); ``wgu`` holds gate and up rows interleaved in
    blocks of 128 when there are whole blocks, else one after the other.  Fused into the GEMM epilogue for bf16 rows."""
    f = wgu.shape[0] // 2
    if x.is_cuda and x.dtype == torch.bfloat16 and f % 128 == 0 and x.shape[1] % 8 == 0:
        return _C().gemm_clamped_glu(x, wgu, limit, alpha)
    gu = F.linear(x, wgu.to(x.dtype))
    if x.is_cuda:
        return _C().mix_clamped_glu(gu, 128 if f % 128 == 0 else f, limit, alpha)
    g, u = split_gate_up(gu.float()) if f % 128 == 0 else gu.float().split(f, -1)
    g = g.clamp(max=limit)
    return (g * torch.sigmoid(alpha * g) * (u.clamp(-limit, limit) + 1)).to(x.dtype)


def linear_silu_glu(x: torch.Tensor, wgu: torch.Tensor) -> torch.Tensor:
    """silu(gate) * up; ``wgu`` laid out as in ``linear_clamped_glu``.  Fused into the GEMM epilogue for bf16 rows — but for few rows of a narrow
    layer, whose 256-row weight tiles would leave most SMs idle: library product, then the gate."""
    f = wgu.shape[0] // 2
    narrow = x.shape[0] <= 128 and wgu.shape[0] < 256 * 74
    if not narrow and x.is_cuda and x.dtype == torch.bfloat16 and f % 128 == 0 and x.shape[1] % 8 == 0:
        return _C().gemm_swiglu(x, wgu, False)[0]
    return silu_glu(F.linear(x, wgu.to(x.dtype)), f)


def silu_glu(gu: torch.Tensor, f: int) -> torch.Tensor:
    if gu.is_cuda:
        return _C().mix_silu_glu(gu, 128 if f % 128 == 0 else f)
    g, u = split_gate_up(gu.float()) if f % 128 == 0 else gu.float().split(f, -1)
    return (F.silu(g) * u).to(gu.dtype)


def poly_norm(z: torch.Tensor, act: torch.Tensor, eps: float) -> torch.Tensor:
    """a N(z) + b N(z^2) + c N(z^3) + e with N(u) = u / sqrt(mean(u^2) + eps) over a row and act = [a, b, c, e]."""
    if z.is_cuda:
        return _C().mix_poly_norm(z, act, eps)
    x = z.float()
    return (act[0] * _rms(x, eps) + act[1] * _rms(x * x, eps) + act[2] * _rms(x ** 3, eps) + act[3]).to(z.dtype)


# --------------------------------------------------------------------------------------------
# parallel blocks: results of the layers so far, input convolutions
# --------------------------------------------------------------------------------------------
@dataclass
class InputConv:
    """h -> h + conv(h) for one or two sublayers that read the same h: weights [taps, ch] (last row: the current token), and the state
    [slots, taps - 1, ch] that both share."""
    w1: torch.Tensor
    w2: torch.Tensor | None
    state: torch.Tensor


@dataclass
class Routed:
    """Rows of ``experts`` in the experts' order; row ``pos[t, j]`` belongs to token t, with ``weight[t, j]`` if there are weights."""
    rows: torch.Tensor
    pos: torch.Tensor
    weight: torch.Tensor | None = None

    def sum(self) -> torch.Tensor:
        r = self.rows.float()[self.pos.long()]
        return r.sum(1) if self.weight is None else (r * self.weight[..., None]).sum(1)


def input_conv(h: torch.Tensor, conv: InputConv | None, b: SpanBatch) -> tuple[torch.Tensor, torch.Tensor | None]:
    """What the two sublayers read (the second is None when there is no second weight)."""
    if conv is None:
        return h, h
    if h.is_cuda:
        out = _C().mix_input_conv(h, conv.w1, conv.w2, conv.state, b.cu, b.start, b.slot, b.seq_of)
        return out[0], (out[1] if conv.w2 is not None else None)
    taps = conv.w1.shape[0]
    out = [None if w is None else torch.empty_like(h) for w in (conv.w1, conv.w2)]
    cu = b.cu.tolist()
    for s in range(b.spans):
        lo, hi = cu[s], cu[s + 1]
        old = conv.state[b.slot[s]] if int(b.start[s]) else torch.zeros_like(conv.state[0])
        full = torch.cat([old, h[lo:hi]]).float()
        for o, w in zip(out, (conv.w1, conv.w2)):
            if o is not None:
                o[lo:hi] = (full[taps - 1:] + sum(w[j] * full[j:j + hi - lo] for j in range(taps))).to(h.dtype)
        conv.state[b.slot[s]] = full[full.shape[0] - (taps - 1):].to(h.dtype)
    return out[0], out[1]


def _fused_conv(conv: InputConv | None, b: SpanBatch) -> tuple:
    """Arguments of the kernels that end in the convolution of single tokens, or nothing."""
    return (None,) * 5 if conv is None or b.seq_of is not None else (conv.w1, conv.w2, conv.state, b.start, b.slot)


def block_embed(ids: torch.Tensor, w: torch.Tensor, slots: int, w_norm: torch.Tensor, eps: float, center: bool, conv: InputConv | None,
                b: SpanBatch) -> tuple[torch.Tensor, tuple]:
    """(results of the layers [slots, T, W] in fp32 with the embedding in the first, what the first layer's sublayers read)."""
    if w.is_cuda:
        past, *h = _C().mix_block_embed(ids, w, slots, w_norm, eps, center, *_fused_conv(conv, b))
        return past, _read(h, conv, b)
    x = F.embedding(ids, w).float()
    past = x.new_empty(slots, *x.shape)
    past[0] = x
    return past, input_conv((_norm(x, eps, center) * w_norm).to(w.dtype), conv, b)


def _read(h: list, conv: InputConv | None, b: SpanBatch) -> tuple:
    if conv is None:
        return h[0], h[0]
    return input_conv(h[0], conv, b) if b.seq_of is not None else (h[0], h[1] if conv.w2 is not None else None)


def block_add(past: torch.Tensor, i: int, y1: torch.Tensor, y2: torch.Tensor | None, routed: Routed | None, s1: torch.Tensor | None,
              s2: torch.Tensor | None, a_prev: torch.Tensor | None, a_cur: torch.Tensor | None, w_next: torch.Tensor | None, eps: float, center: bool,
              conv: InputConv | None, b: SpanBatch, want_x: bool = False) -> tuple[torch.Tensor | None, tuple]:
    """Layer ``i`` of a stack of parallel blocks:  X = x + s1 y1 + s2 (y2 + sum of its routed rows)  with x = sum_j a_prev[j] past[j] (past[0]
    without ``a_prev``), then x' = sum_j a_cur[j] past[j] + a_cur[i + 1] X.  X goes to past[i + 1] (without averages: to past[0], and x' = X).
    Returns (x' in fp32 if wanted, what the next layer's sublayers read: norm(x') * w_next through ``conv``)."""
    if y1.is_cuda:
        rows, pos = (routed.rows, routed.pos) if routed is not None else (None, None)
        x, *h = _C().mix_block_add(past, i, y1, y2, rows, pos, s1, s2, a_prev, a_cur, w_next, eps, center, want_x, *_fused_conv(conv, b))
        return (x if want_x else None), ((None, None) if w_next is None else _read(h, conv, b))
    x = past[0].clone() if a_prev is None else torch.einsum("j,jtw->tw", a_prev, past[:i + 1])
    y = y1.float() if s1 is None else y1.float() * s1
    if y2 is not None or routed is not None:
        f = (0 if y2 is None else y2.float()) + (0 if routed is None else routed.sum())
        y = y + (f if s2 is None else f * s2)
    x = x + y
    past[0 if a_cur is None else i + 1] = x
    if a_cur is not None:
        x = torch.einsum("j,jtw->tw", a_cur, past[:i + 2])
    return (x if want_x else None), ((None, None) if w_next is None else input_conv((_norm(x, eps, center) * w_next).to(y1.dtype), conv, b))


# --------------------------------------------------------------------------------------------
# experts
# --------------------------------------------------------------------------------------------
TILE = 128              # rows of the expert kernels' tiles: every expert's rows start on one


def experts(h: torch.Tensor, router: torch.Tensor, wgu: torch.Tensor, wd: torch.Tensor, top: int, clamp: tuple[float, float] | None = None,
            softmax: bool = False) -> Routed:
    """Gated experts.  Token t goes to the ``top`` experts with the largest scores: s = sigmoid(router h), and each reads s h — or, with ``softmax``,
    s = softmax(router h) over all experts, each reads h and its result counts with s over the sum of the chosen ones (+ 1e-20).  The gate is
    silu(gate) * up, with ``clamp`` = (limit, alpha) that of ``linear_clamped_glu``.  wgu [E * 2 F, W] holds every expert's gate and up rows as in
    ``linear_silu_glu``, wd [E * W, F].  No host synchronisation."""
    e, width = router.shape[0], h.shape[1]
    f = wgu.shape[0] // (2 * e)
    logits = linear_f32(h, router)
    if h.is_cuda:
        C = _C()
        pick, score, rank, plan = C.mix_route(logits, top, _counter(h.device, e + 1, "route"), softmax)
        rows, pos = C.mix_expert_rows(h, pick, None if softmax else score, rank, plan, e)
        limit, alpha = clamp or (0.0, 0.0)
        if h.dtype == torch.bfloat16 and f % 128 == 0 and width % 8 == 0:
            out = C.gemm_experts(C.gemm_experts(rows, wgu, plan, e, 1 if clamp is None else 2, limit, alpha), wd, plan, e, 0)
        else:
            gu = C.mix_expert_gemm(rows, wgu, plan, e)
            blk = 128 if f % 128 == 0 else f
            out = C.mix_expert_gemm(silu_glu(gu, f) if clamp is None else C.mix_clamped_glu(gu, blk, limit, alpha), wd, plan, e)
        return Routed(out, pos, score if softmax else None)
    score, pick = torch.topk(torch.softmax(logits, -1) if softmax else torch.sigmoid(logits), top, dim=-1)
    if softmax:
        score = score / (score.sum(-1, keepdim=True) + 1e-20)
    rows = h.new_empty(h.shape[0] * top, width)
    pos = torch.arange(rows.shape[0]).reshape(-1, top)
    x = h[:, None].expand(-1, top, -1) if softmax else (h.float()[:, None] * score[..., None]).to(h.dtype)
    for j in range(e):
        t, k = (pick == j).nonzero(as_tuple=True)
        if t.numel():
            up = wgu[j * 2 * f:(j + 1) * 2 * f]
            a = silu_glu(F.linear(x[t, k], up), f) if clamp is None else linear_clamped_glu(x[t, k], up, *clamp)
            rows[pos[t, k]] = F.linear(a, wd[j * width:(j + 1) * width])
    return Routed(rows, pos, score if softmax else None)


# --------------------------------------------------------------------------------------------
# residual streams
# --------------------------------------------------------------------------------------------
def streams_embed(ids: torch.Tensor, w: torch.Tensor, scale: float, streams: int, win: torch.Tensor, w_norm: torch.Tensor, eps: float) -> tuple:
    """(streams in fp32 — one row per token while all of them are equal: [T, 1, W] — and what the first sublayer reads, the norm of sum_s win[s] x)."""
    if w.is_cuda:
        return tuple(_C().mix_streams_embed(ids, w, scale, streams, win, w_norm, eps))
    x = F.embedding(ids, w).float() * scale
    return x[:, None], (_rms(x * win.sum(), eps) * w_norm).to(w.dtype)


def _streams_after(x, y, bias, routed, mix, out):
    t = (0 if y is None else y.float()) + (0 if bias is None else bias) + (0 if routed is None else routed.sum())
    return torch.einsum("sr,tsw->trw", mix, x.expand(-1, mix.shape[0], -1)) + out[:, None] * t[:, None]


def streams_add(x: torch.Tensor, y: torch.Tensor | None, bias: torch.Tensor | None, routed: Routed | None, mix: torch.Tensor, out: torch.Tensor,
                win: torch.Tensor, w_norm: torch.Tensor, eps: float) -> tuple[torch.Tensor, torch.Tensor]:
    """End of a sublayer and beginning of the next:  X_t = sum_s mix[s, t] x_s + out[t] (y + bias + weighted routed rows)  in fp32 [T, streams, W] (in
    place where x has that shape), and norm(sum_t win[t] X_t) * w_norm in y's dtype."""
    if x.is_cuda:
        return tuple(_C().mix_streams_add(x, y, bias, *_routed(routed), mix, out, win, w_norm, eps, False))
    x = _streams_after(x, y, bias, routed, mix, out)
    return x, (_rms(torch.einsum("s,tsw->tw", win, x), eps) * w_norm).to((y if y is not None else routed.rows).dtype)


def streams_sum(x: torch.Tensor, y: torch.Tensor | None, bias: torch.Tensor | None, routed: Routed | None, mix: torch.Tensor, out: torch.Tensor,
                w_norm: torch.Tensor | None, eps: float) -> tuple[torch.Tensor, torch.Tensor | None]:
    """End of the last sublayer: (sum of the streams in fp32, its norm when there is a weight)."""
    if x.is_cuda:
        x, h = _C().mix_streams_add(x, y, bias, *_routed(routed), mix, out, None, w_norm, eps, True)
        return x, (h if w_norm is not None else None)
    x = _streams_after(x, y, bias, routed, mix, out).sum(1)
    return x, (None if w_norm is None else (_rms(x, eps) * w_norm).to((y if y is not None else routed.rows).dtype))


def _routed(r: Routed | None) -> tuple:
    return (None, None, None) if r is None else (r.rows, r.pos, r.weight)


# --------------------------------------------------------------------------------------------
# causal convolution with carried taps
# --------------------------------------------------------------------------------------------
def conv_silu(x: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None, state: torch.Tensor, b: SpanBatch) -> torch.Tensor:
    """silu(causal conv) per channel; w [taps, ch] (last row: the current token), state [slots, taps - 1, ch]."""
    if x.is_cuda:
        return _C().mix_conv(x, w, bias, state, b.cu, b.start, b.slot, b.seq_of)
    taps = w.shape[0]
    out = torch.empty_like(x)
    cu = b.cu.tolist()
    for s in range(b.spans):
        lo, hi = cu[s], cu[s + 1]
        old = state[b.slot[s]] if int(b.start[s]) else torch.zeros_like(state[0])
        full = torch.cat([old, x[lo:hi]]).float()
        y = (0 if bias is None else bias) + sum(w[j] * full[j:j + hi - lo] for j in range(taps))
        out[lo:hi] = F.silu(y).to(x.dtype)
        state[b.slot[s]] = full[full.shape[0] - (taps - 1):].to(state.dtype)
    return out


# --------------------------------------------------------------------------------------------
# gated linear recurrences
# --------------------------------------------------------------------------------------------
SSD, MLSTM, DELTA, DECAY, GLA = range(5)


@dataclass
class Gates:
    """Raw gate projections (fp32 [T, H], ``GLA``: [T, H * N]) and per-head constants of a recurrence."""
    g0: torch.Tensor | None = None
    g1: torch.Tensor | None = None
    b0: torch.Tensor | None = None
    b1: torch.Tensor | None = None
    a_log: torch.Tensor | None = None
    d_skip: torch.Tensor | None = None
    cap: float = 1.0                    # GLA: tau
    raw: bool = False                   # DECAY: q, k and v are still to be silu-activated (single tokens only)


CHUNK_MIN = 8           # spans shorter than this go through the token-by-token kernel
TC_MIN = 65             # from here on the 128-token tcgen05 chunks pay


def scan(mode: int, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gates: Gates, qscale: float, cache: dict, b: SpanBatch) -> torch.Tensor:
    """S_t = keep_t S_(t-1) + add_t k_t v_t^T,  y_t = S_t^T (qscale q_t), over the spans of ``b``.

    ``SSD``: add = softplus(g0 + b0), keep = exp(-exp(a_log) add), y += d_skip v.  ``MLSTM``: capped log gates with a running
    maximum and a normaliser.  ``DELTA``: the gated delta rule on unit vectors k' = k / |k|, q' = q / |q| (1e-6 under the root): keep =
    exp(-exp(a_log) softplus(g0 + b0)) and the write is k' u^T with u = sigmoid(g1) (v - keep S^T k').  ``DECAY``: add = 1, keep = exp(a_log).
    ``GLA``: add = 1 and a keep for every state row, sigmoid(g0 + b0)^(1 / cap).  q / k [T, groups * N] (consecutive heads share a group), v [T, H * V], cache["S"] [slots, H, N, V]
    (+ "n" [slots, H, N], "m" [slots, H])."""
    if not v.is_cuda:
        return _scan_cpu(mode, q, k, v, gates, qscale, cache, b)
    S, H, N = cache["S"], cache["S"].shape[1], cache["S"].shape[2]
    ctr = _counter(v.device, b.spans * H)
    out = torch.empty(v.shape, device=v.device, dtype=v.dtype)

    def run(lo: int, hi: int, form: int) -> None:       # 0: token by token, 1: one token per span, 2 / 3: chunked
        _C().mix_scan_(mode, q, k, v, gates.g0, gates.g1, gates.b0, gates.b1, gates.a_log, gates.d_skip, qscale, gates.cap, gates.raw, S, cache.get("n"),
                       cache.get("m"), b.cu[lo:hi + 1], b.start[lo:hi], b.slot[lo:hi], ctr, form, out)

    chunk = v.dtype == torch.bfloat16 and b.max_long >= CHUNK_MIN
    if b.n_long and mode == DELTA and chunk and _C().mix_delta_chunk_ok(q, k, v, S):
        _C().mix_delta_chunk_(q, k, v, gates.g0, gates.g1, gates.b0, gates.a_log, qscale, S, b.cu[:b.n_long + 1], b.start[:b.n_long],
                              b.slot[:b.n_long], ctr, out)
    elif b.n_long and mode == GLA and chunk and _C().mix_gla_chunk_(q, k, v, gates.g0, gates.b0, qscale, gates.cap, S, b.cu[:b.n_long + 1], b.start[:b.n_long],
                                                                    b.slot[:b.n_long], ctr, out):
        pass
    elif b.n_long:
        chunk = chunk and mode not in (DELTA, GLA) and _C().mix_chunk_supported(N)
        run(0, b.n_long, (3 if b.max_long >= TC_MIN else 2) if chunk else 0)
    if b.n_long < b.spans:
        run(b.n_long, b.spans, 1)
    return out


def _scan_cpu(mode, q, k, v, g: Gates, qscale, cache, b: SpanBatch):
    S_pool = cache["S"]
    H, N, V = S_pool.shape[1:]
    rep = H // (q.shape[1] // N)
    out = torch.empty_like(v)
    cu = b.cu.tolist()
    for s in range(b.spans):
        sl, fresh = int(b.slot[s]), int(b.start[s]) == 0
        S = torch.zeros_like(S_pool[0]) if fresh else S_pool[sl].clone()
        if mode == MLSTM:
            n = torch.zeros_like(cache["n"][0]) if fresh else cache["n"][sl].clone()
            m = torch.zeros_like(cache["m"][0]) if fresh else cache["m"][sl].clone()
        for t in range(cu[s], cu[s + 1]):
            qt = q[t].float().reshape(-1, N).repeat_interleave(rep, 0)
            kt = k[t].float().reshape(-1, N).repeat_interleave(rep, 0)
            if mode == DELTA:
                qt, kt = (x * torch.rsqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6) for x in (qt, kt))
            vt = v[t].float().reshape(H, V)
            if g.raw:
                qt, kt, vt = (F.silu(x).to(v.dtype).float() for x in (qt, kt, vt))
            qt = qt * qscale
            if mode == DECAY:
                keep, add = torch.exp(g.a_log), torch.ones(H)
            elif mode == GLA:
                keep, add = torch.exp(F.logsigmoid(g.g0[t] + g.b0) / g.cap).reshape(H, N), torch.ones(H)
            elif mode in (SSD, DELTA):
                add = F.softplus(g.g0[t] + g.b0, threshold=1e9)
                keep = torch.exp(-torch.exp(g.a_log) * add)
            else:
                gi = g.cap * torch.tanh((g.g0[t] + g.b0) / g.cap)
                gf = F.logsigmoid(g.cap * torch.tanh((g.g1[t] + g.b1) / g.cap))
                m2 = torch.maximum(gf + m, gi)
                keep, add, m = torch.exp(gf + m - m2), torch.exp(gi - m2), m2
                n = keep[:, None] * n + add[:, None] * kt
            if mode == DELTA:
                S = keep[:, None, None] * S
                u = torch.sigmoid(g.g1[t])[:, None] * (vt - torch.einsum("hnv,hn->hv", S, kt))
                S = S + kt[:, :, None] * u[:, None, :]
            else:
                S = keep.reshape(H, -1, 1) * S + (add[:, None] * kt)[:, :, None] * vt[:, None, :]
            y = torch.einsum("hnv,hn->hv", S, qt)
            if mode == SSD:
                y = y + g.d_skip[:, None] * vt
            elif mode == MLSTM:
                y = y / (torch.maximum((n * qt).sum(-1).abs(), torch.exp(-m)) + 1e-6)[:, None]
            out[t] = y.reshape(-1).to(v.dtype)
        S_pool[sl] = S
        if mode == MLSTM:
            cache["n"][sl], cache["m"][sl] = n, m
    return out


def selective_scan(x: torch.Tensor, dt: torch.Tensor, bm: torch.Tensor, cm: torch.Tensor, z: torch.Tensor, dt_bias: torch.Tensor, a_neg: torch.Tensor,
                   d_skip: torch.Tensor, state: torch.Tensor, b: SpanBatch) -> torch.Tensor:
    """Per channel c and state n, with d = softplus(dt + dt_bias):  S[c, n] = exp(d_c a_neg[c, n]) S[c, n] + d_c x_c B_n,
    y_c = sum_n S[c, n] C_n + d_skip_c x_c; returns y silu(z).  x, z [T, C], dt fp32 [T, C], bm, cm [T, N], state [slots, C, N]."""
    if x.is_cuda:
        return _C().mix_selective(x, dt, bm, cm, z, dt_bias, a_neg, d_skip, state, b.cu, b.start, b.slot, b.n_long)
    out = torch.empty_like(x)
    cu = b.cu.tolist()
    for s in range(b.spans):
        sl = int(b.slot[s])
        S = state[sl].clone() if int(b.start[s]) else torch.zeros_like(state[0])
        for t in range(cu[s], cu[s + 1]):
            xt, d = x[t].float(), F.softplus(dt[t] + dt_bias, threshold=1e9)
            S = torch.exp(d[:, None] * a_neg) * S + (d * xt)[:, None] * bm[t].float()
            out[t] = ((S @ cm[t].float() + d_skip * xt) * F.silu(z[t].float())).to(x.dtype)
        state[sl] = S
    return out


# --------------------------------------------------------------------------------------------
# latent attention
# --------------------------------------------------------------------------------------------
def rope_frequencies(dims: int, base: float, device) -> torch.Tensor:
    """base^(-2 i / dims), i < dims / 2, double precision (angles are reduced before the fp32 sine / cosine)."""
    return torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float64, device=device)


def scaled_frequencies(dims: int, base: float, scaling: dict | None, device) -> torch.Tensor:
    """``rope_frequencies`` with Llama 3.1's scaling {"factor", "low", "high", "original"}: wavelengths above original / low are stretched by
    ``factor``, those below original / high stay, the ones between are blended."""
    f = rope_frequencies(dims, base, "cpu")
    if scaling:
        s = ((scaling["original"] * f / (2 * math.pi) - scaling["low"]) / (scaling["high"] - scaling["low"])).clamp(0, 1)
        f = (1 - s) * f / scaling["factor"] + s * f
    return f.to(device)


def _rotate(x: torch.Tensor, freq: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
    a = torch.outer(pos.double(), freq)
    c, s = a.cos().float(), a.sin().float()
    if x.dim() == 3:
        c, s = c[:, None], s[:, None]
    u, v = x.float().chunk(2, -1)
    return torch.cat([u * c - v * s, v * c + u * s], -1).to(x.dtype)


def latent_prep(a: torch.Tensor, wq: torch.Tensor, wkv: torch.Tensor, freq: torch.Tensor, pool: torch.Tensor, b: SpanBatch, eps: float,
                want_entry: bool) -> tuple[torch.Tensor, torch.Tensor | None]:
    """Rows [query latent | key-value latent | shared rotary key] -> normed query latent; the cache row [normed latent | rotated key] of
    every token is written to ``pool`` and also returned when asked for."""
    if a.is_cuda:
        cq, en = _C().mix_latent_prep(a, wq, wkv, freq, b.pos, b.kv_slot, pool, eps, want_entry)
        return cq, en if want_entry else None
    qr, r, rd = wq.numel(), wkv.numel(), 2 * freq.numel()
    cq = (_rms(a[:, :qr].float(), eps) * wq).to(a.dtype)
    c = (_rms(a[:, qr:qr + r].float(), eps) * wkv).to(a.dtype)
    en = torch.cat([c, _rotate(a[:, qr + r:qr + r + rd], freq, b.pos)], -1)
    pool.view(-1, r + rd)[b.kv_slot] = en
    return cq, en


def rope_(q: torch.Tensor, d: int, freq: torch.Tensor, pos: torch.Tensor) -> None:
    """Rotate columns [d, d + 2 * freq.numel()) of every head of q [T, H, *] in place."""
    if q.is_cuda:
        _C().mix_rope_(q, d, freq, pos)
        return
    rd = 2 * freq.numel()
    q[..., d:d + rd] = _rotate(q[..., d:d + rd], freq, pos)


def _splits(rows: int, heads: int, max_len: int) -> int:
    ctas = rows * ((heads + 31) // 32)
    return max(1, min((2 * 148 + ctas - 1) // ctas, max(1, max_len // 256), 32))


def latent_attention(q_lat: torch.Tensor, q: torch.Tensor, d: int, pool: torch.Tensor, table: torch.Tensor, seq_of: torch.Tensor | None,
                     kv_len: torch.Tensor, sink: torch.Tensor | None, scale: float, max_len: int) -> torch.Tensor:
    """Absorbed form over the paged pool: q_lat [H, R, r], q [R, H, *] (rotated part at column d) -> softmax-weighted latents [H, R, r];
    ``sink`` [H] adds exp(sink) to the denominator."""
    h, rows, r = q_lat.shape
    if q.is_cuda:
        tc = q.dtype == torch.bfloat16 and _C().mix_latent_tc_ok(r, pool.shape[-1] - r)
        return _C().mix_latent(q_lat, q, d, pool, table, seq_of, kv_len, sink, scale, _splits(rows, h, max_len), tc)
    rd = pool.shape[-1] - r
    out = torch.zeros_like(q_lat)
    for i in range(rows):
        n = int(kv_len[i])
        if n == 0:
            continue
        pages = table[int(seq_of[i]) if seq_of is not None else i, : (n + PAGE - 1) // PAGE].long()
        kv = pool.view(-1, PAGE, r + rd)[pages].reshape(-1, r + rd)[:n].float()
        s = (q_lat[:, i].float() @ kv[:, :r].T + q[i, :, d:d + rd].float() @ kv[:, r:].T) * scale
        if sink is not None:
            s = torch.cat([s, sink[:, None]], -1)
        p = torch.softmax(s, -1)[:, :n]
        out[:, i] = (p @ kv[:, :r]).to(out.dtype)
    return out


def sink_varlen_ok(kw: int, vw: int) -> bool:
    """Widths that the packed kernel takes."""
    return (kw, vw) in ((64, 64), (64, 128), (128, 64), (128, 128), (192, 128))


def sink_attention_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_q: torch.Tensor, cu_k: torch.Tensor, scale: float,
                          sink: torch.Tensor | None) -> torch.Tensor:
    """Causal (bottom-right aligned) attention of packed spans, with a sink: the tcgen05 kernel, widths of ``sink_varlen_ok``, bf16."""
    return _C().attn_fwd(q, k, v, cu_q, cu_k, scale, True, False, None, sink)[0]


# --------------------------------------------------------------------------------------------
# grouped-query attention in a sliding window with kept first tokens
# --------------------------------------------------------------------------------------------
def _rotate_pairs(x: torch.Tensor, freq: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
    """x [T, heads, d]: neighbours (2 i, 2 i + 1) of the first entries turned by pos * freq[i]."""
    a = torch.outer(pos.double(), freq)
    c, s = a.cos().float()[:, None], a.sin().float()[:, None]
    y, n = x.clone(), 2 * freq.numel()
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y[..., 0:n:2], y[..., 1:n:2] = u * c - v * s, v * c + u * s
    return y


def qk_prep(p: torch.Tensor, heads: int, dim: int, wq: torch.Tensor, wk: torch.Tensor, freq: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor,
            b: SpanBatch, eps: float, want_kv: bool) -> tuple[torch.Tensor, tuple | None]:
    """Rows [queries | keys] as projected -> queries [T, heads, width], RMS-normed over the whole row and rotated; the keys treated alike go to
    ``k_pool`` and, as projected, to ``v_pool`` ([pages, key heads, PAGE, width], zeros beyond ``dim``).  Packed keys and values [T, key heads,
    width] are returned too when asked for."""
    g, width = k_pool.shape[1], k_pool.shape[3]
    if p.is_cuda:
        q, k, v = _C().mix_qk_prep(p, heads, dim, wq, wk, freq, b.pos, b.kv_slot, k_pool, v_pool, eps, want_kv)
        return q, ((k, v) if want_kv else None)
    t = p.shape[0]
    raw = p[:, heads * dim:(heads + g) * dim]
    q = _rotate_pairs((_rms(p[:, :heads * dim].float(), eps) * wq).reshape(t, heads, dim), freq, b.pos)
    k = _rotate_pairs((_rms(raw.float(), eps) * wk).reshape(t, g, dim), freq, b.pos)
    q, k, v = (F.pad(x.to(p.dtype), (0, width - dim)) for x in (q, k, raw.reshape(t, g, dim)))
    page, off = b.kv_slot // PAGE, b.kv_slot % PAGE
    k_pool[page, :, off], v_pool[page, :, off] = k, v
    return q, ((k, v) if want_kv else None)


def gather_keys(k_pool: torch.Tensor, v_pool: torch.Tensor, rows: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """Keys and values of flat cache rows, [rows, key heads, width] each."""
    if k_pool.is_cuda:
        return tuple(_C().mix_gather_keys(k_pool, v_pool, rows))
    return k_pool[rows // PAGE, :, rows % PAGE], v_pool[rows // PAGE, :, rows % PAGE]


def window_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, table: torch.Tensor, seq_of: torch.Tensor | None, kv_len: torch.Tensor,
                     scale: float, window: int, keep_first: int, max_len: int) -> torch.Tensor:
    """Paged form, one query row [heads, width] per entry of ``kv_len``: the row's own token is its last key; it sees the last ``window``
    keys and the first ``keep_first``."""
    rows, h, width = q.shape
    g = k_pool.shape[1]
    if q.is_cuda:
        if q.dtype == torch.bfloat16 and width in (64, 128) and h // g <= 16 and seq_of is None:
            from .functional import paged_decode_attention

            return paged_decode_attention(q.reshape(rows, h * width), k_pool, v_pool, table, kv_len, h, g, width, scale,
                                          max_len=min(max_len, window + keep_first + 2 * PAGE), window=window, keep_first=keep_first).view(rows, h, width)
        return _C().mix_window_attention(q, k_pool, v_pool, table, seq_of, kv_len, scale, window, keep_first)
    out = torch.zeros_like(q)
    for i in range(rows):
        n = int(kv_len[i])
        if n == 0:
            continue
        pages = table[int(seq_of[i]) if seq_of is not None else i, : (n + PAGE - 1) // PAGE].long()
        j = torch.arange(n)
        j = j[(j >= n - window) | (j < keep_first)]
        k, v = (x[pages[j // PAGE], :, j % PAGE].float().repeat_interleave(h // g, 1) for x in (k_pool, v_pool))
        s = torch.softmax(torch.einsum("hd,jhd->hj", q[i].float(), k) * scale, -1)
        out[i] = torch.einsum("hj,jhd->hd", s, v).to(q.dtype)
    return out


def window_attention_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_q: torch.Tensor, cu_k: torch.Tensor, scale: float, window: int,
                            keep_first: int) -> torch.Tensor:
    """Packed spans, bottom-right aligned: the tcgen05 kernel, width 64 or 128, bf16."""
    return _C().attn_fwd(q, k, v, cu_q, cu_k, scale, True, False, None, None, window, keep_first)[0]


# --------------------------------------------------------------------------------------------
# attention with rotated values and a sink
# --------------------------------------------------------------------------------------------
def turn_prep(p: torch.Tensor, bias: torch.Tensor, heads: int, dim: int, vdim: int, freq: torch.Tensor, vfreq: torch.Tensor, k_pool: torch.Tensor,
              v_pool: torch.Tensor, b: SpanBatch, eps: float, want_kv: bool) -> tuple[torch.Tensor, tuple | None]:
    """Rows [queries: heads x dim | keys: groups x dim | values: groups x vdim] as projected, without their ``bias`` -> queries [T, heads, key width],
    rotated (entries i and i + freq.numel()) and divided by their root mean square; the keys treated alike go to ``k_pool`` ([pages, groups, PAGE, key
    width]), the values, rotated over all of ``vdim``, to ``v_pool``.  Packed keys and values are returned too when asked for."""
    g, kw, vw = k_pool.shape[1], k_pool.shape[3], v_pool.shape[3]
    if p.is_cuda:
        q, k, v = _C().mix_turn_prep(p, bias, heads, dim, vdim, freq, vfreq, b.pos, b.kv_slot, k_pool, v_pool, eps, want_kv)
        return q, ((k, v) if want_kv else None)
    t, nq = p.shape[0], heads * dim
    x = p.float() + bias

    def turned(y, f):
        n = 2 * f.numel()
        return torch.cat([_rotate(y[..., :n], f, b.pos), y[..., n:]], -1)

    q, k = (_rms(turned(y.reshape(t, -1, dim), freq), eps).to(p.dtype) for y in (x[:, :nq], x[:, nq:nq + g * dim]))
    v = turned(x[:, nq + g * dim:].reshape(t, g, vdim), vfreq).to(p.dtype)
    q, k, v = F.pad(q, (0, kw - dim)), F.pad(k, (0, kw - dim)), F.pad(v, (0, vw - vdim))
    page, off = b.kv_slot // PAGE, b.kv_slot % PAGE
    k_pool[page, :, off], v_pool[page, :, off] = k, v
    return q, ((k, v) if want_kv else None)


def turn_back(o: torch.Tensor, gate: torch.Tensor, vfreq: torch.Tensor, pos: torch.Tensor, scale: float, out: torch.Tensor) -> torch.Tensor:
    """o [T, heads, value width]: entries (m, m + vdim / 2) of every head turned by -pos * vfreq[m], times scale * sigmoid(gate) -> out [T, heads * vdim]."""
    if o.is_cuda:
        _C().mix_turn_back(o, gate, vfreq, pos, scale, out)
        return out
    x = _rotate(o[..., :2 * vfreq.numel()].float(), -vfreq, pos).reshape(o.shape[0], -1)
    return out.copy_((x * torch.sigmoid(gate.float()) * scale).to(o.dtype))


def sink_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, table: torch.Tensor, seq_of: torch.Tensor | None, kv_len: torch.Tensor,
                   scale: float, sink: torch.Tensor, max_len: int) -> torch.Tensor:
    """Paged form, one query row [heads, key width] per entry of ``kv_len`` (its own token is its last key) -> [rows, heads, value width]; ``sink``
    [heads] adds exp(sink) to the denominator."""
    rows, h, kw = q.shape
    g, vw = k_pool.shape[1], v_pool.shape[3]
    if q.is_cuda:
        if q.dtype == torch.bfloat16 and sink_varlen_ok(kw, vw) and h // g <= 16 and seq_of is None:
            from .functional import _auto_splits

            return _C().sink_decode(q, k_pool, v_pool, table, kv_len, scale, _auto_splits(rows, g, max_len), sink)
        return _C().mix_sink_attention(q, k_pool, v_pool, table, seq_of, kv_len, scale, sink)
    out = q.new_zeros(rows, h, vw)
    for i in range(rows):
        n = int(kv_len[i])
        if n == 0:
            continue
        pages = table[int(seq_of[i]) if seq_of is not None else i, : (n + PAGE - 1) // PAGE].long()
        j = torch.arange(n)
        k, v = (x[pages[j // PAGE], :, j % PAGE].float().repeat_interleave(h // g, 1) for x in (k_pool, v_pool))
        s = torch.cat([torch.einsum("hd,jhd->hj", q[i].float(), k) * scale, sink[:, None]], -1)
        out[i] = torch.einsum("hj,jhd->hd", torch.softmax(s, -1)[:, :n], v).to(q.dtype)
    return out


# --------------------------------------------------------------------------------------------
# differential attention: two softmax maps per head over the same values
# --------------------------------------------------------------------------------------------
@dataclass
class MapMix:
    """o = a1 - lam a2,  o / sqrt(mean(o^2) + eps) * (1 - diff)  over the ``vdim`` values of a head."""
    lam: torch.Tensor           # [1] fp32
    diff: float
    eps: float
    vdim: int
    dim: int                    # of a query or key, without padding

    def __call__(self, a1: torch.Tensor, a2: torch.Tensor) -> torch.Tensor:
        return _rms((a1 - self.lam * a2)[..., :self.vdim], self.eps) * (1 - self.diff)


def query_map_width(kw: int, dtype: torch.dtype) -> int:
    """Width of a map's query at run time: the keys' — or 64 for bf16 keys of width 32, whose two maps share one 64-wide row: the query of map m
    then lies at column 32 m, zeros beside it."""
    return 64 if kw == 32 and dtype == torch.bfloat16 else kw


def map_prep(p: torch.Tensor, bias: torch.Tensor, heads: int, dim: int, vdim: int, wq: torch.Tensor, wk: torch.Tensor, freq: torch.Tensor,
             k_pool: torch.Tensor, v_pool: torch.Tensor, b: SpanBatch, eps: float, want_kv: bool) -> tuple[torch.Tensor, tuple | None]:
    """Rows [queries: heads x 2 maps x dim | keys: groups x 2 maps x dim | values: groups x vdim] as projected, without their ``bias`` -> queries
    [T, 2 heads, query_map_width], RMS-normed per map and rotated (entries i and i + freq.numel()); the keys treated alike go to ``k_pool``
    ([pages, groups, PAGE, 2 key widths]) and the values to ``v_pool``.  Packed keys and values are returned too when asked for."""
    g, kw, vw = k_pool.shape[1], k_pool.shape[3] // 2, v_pool.shape[3]
    qw = query_map_width(kw, p.dtype)
    if p.is_cuda:
        q, k, v = _C().mix_map_prep(p, bias, heads, dim, vdim, wq, wk, freq, b.pos, b.kv_slot, k_pool, v_pool, eps, want_kv, qw)
        return q, ((k, v) if want_kv else None)
    t, nq = p.shape[0], 2 * heads * dim
    x = p.float()[:, :nq + 2 * g * dim + g * vdim] + bias
    a = torch.outer(b.pos.double(), freq)
    c, s = a.cos().float()[:, None], a.sin().float()[:, None]

    def turned(y, w):
        y = _rms(y.reshape(t, -1, dim), eps) * w
        n = freq.numel()
        u, v, rest = y[..., :n], y[..., n:2 * n], y[..., 2 * n:]
        return torch.cat([u * c - v * s, v * c + u * s, rest], -1).to(p.dtype)

    q, k = turned(x[:, :nq], wq), F.pad(turned(x[:, nq:nq + 2 * g * dim], wk), (0, kw - dim)).reshape(t, g, 2 * kw)
    v = F.pad(x[:, nq + 2 * g * dim:].reshape(t, g, vdim), (0, vw - vdim)).to(p.dtype)
    if qw == kw:
        q = F.pad(q, (0, qw - dim))
    else:
        q = torch.stack([F.pad(q[:, m::2], (m * kw, qw - m * kw - dim)) for m in range(2)], 2).reshape(t, 2 * heads, qw)
    page, off = b.kv_slot // PAGE, b.kv_slot % PAGE
    k_pool[page, :, off], v_pool[page, :, off] = k, v
    return q, ((k, v) if want_kv else None)


def map_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, table: torch.Tensor, seq_of: torch.Tensor | None, kv_len: torch.Tensor,
                  scale: float, window: int, mix: MapMix, max_len: int) -> torch.Tensor:
    """Paged form, one query row per entry of ``kv_len`` (its own token is its last key, it sees the last ``window``): [rows, heads * vdim]."""
    rows, h, qw = q.shape[0], q.shape[1] // 2, q.shape[2]
    g, kw = k_pool.shape[1], k_pool.shape[3] // 2
    if q.is_cuda:
        if q.dtype == torch.bfloat16 and _C().map_decode_ok(kw, v_pool.shape[3], h // g) and seq_of is None:
            from .functional import _auto_splits

            return _C().map_decode(q, k_pool, v_pool, table, kv_len, scale, _auto_splits(rows, g, min(max_len, window + 2 * PAGE)), window, mix.lam, mix.diff,
                                   mix.eps, mix.vdim)
        return _C().mix_map_attention(q, k_pool, v_pool, table, seq_of, kv_len, scale, window, mix.lam, mix.diff, mix.eps, mix.vdim, mix.dim)
    out = q.new_zeros(rows, h, mix.vdim)
    for i in range(rows):
        n = int(kv_len[i])
        if n == 0:
            continue
        pages = table[int(seq_of[i]) if seq_of is not None else i, : (n + PAGE - 1) // PAGE].long()
        j = torch.arange(max(0, n - window), n)
        k, v = (x[pages[j // PAGE], :, j % PAGE].float().repeat_interleave(h // g, 1) for x in (k_pool, v_pool))
        a = []
        for m in range(2):
            km = k if qw != kw else k[..., m * kw:(m + 1) * kw]
            p = torch.softmax(torch.einsum("hd,jhd->hj", q[i, m::2].float(), km) * scale, -1)
            a.append(torch.einsum("hj,jhd->hd", p, v))
        out[i] = mix(*a).to(q.dtype)
    return out.reshape(rows, -1)


def map_attention_varlen(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_q: torch.Tensor, cu_k: torch.Tensor, scale: float, window: int,
                         mix: MapMix) -> torch.Tensor:
    """Packed spans, bottom-right aligned, q [T, 2 heads, width], k [Tk, groups, 2 key widths], v [Tk, groups, value width]: the tcgen05 kernel
    with both maps of a head in one CTA and their difference in its epilogue -> [T, heads * vdim] (bf16)."""
    return _C().map_attn_fwd(q, k, v, cu_q, cu_k, scale, window, mix.lam, mix.diff, mix.eps, mix.vdim)
