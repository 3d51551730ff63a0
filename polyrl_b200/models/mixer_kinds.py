"""Mixers of ``hybrid.py`` that describe themselves: one ``Kind`` per mixer with its sizes, parameters, caches and step.

  ``turn``       grouped-query attention whose values are rotated like keys and whose outputs are turned back; queries and keys rotated
                 (rotate-half) and divided by their root mean square, a softmax sink per head, an element-wise sigmoid gate, biases
  ``decay``      linear attention with one constant decay per head on silu-activated queries, keys and values; one norm over all heads,
                 sigmoid gate
  ``gla``        gated linear attention: a decay for every key channel from a low-rank projection; norm per head, silu gate
  ``selective``  Mamba's selective scan: a state per channel, step sizes and input / output maps projected from the convolved input
  ``pair``       two of the mixers in ``PAIRABLE`` on the same input, a weighted sum of their outputs: one input and one output product

A mixer's stored parameters are named as in ``specs``; ``prepare`` turns them into what the step reads.  Caches are described by
``Slab``s, from which sizes in bytes and the tensors follow.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Callable

import torch
import torch.nn.functional as F

from .. import ops
from ..ops import mixers as M


def pad8(n: int) -> int:
    return (n + 7) // 8 * 8


@dataclass(frozen=True)
class Slab:
    """One cache tensor: ``shape`` behind the page or slot index; ``paged``: [blocks, heads, PAGE, width], shape = (heads, width)."""
    shape: tuple
    paged: bool = False
    fp32: bool = False

    def make(self, num_blocks: int, num_slots: int, device, dtype: torch.dtype) -> torch.Tensor:
        if self.paged:
            return torch.zeros(num_blocks, self.shape[0], M.PAGE, self.shape[1], device=device, dtype=dtype)
        return torch.zeros(num_slots, *self.shape, device=device, dtype=torch.float32 if self.fp32 else dtype)

    def bytes(self, element: int) -> int:
        return math.prod(self.shape) * (4 if self.fp32 else element)


@dataclass(frozen=True)
class Kind:
    fits: Callable          # sizes -> bool
    specs: Callable         # (sizes, width) -> [(name, shape)]
    prepare: Callable       # (sizes, stored, dtype, is_cuda) -> run-time tensors ("wo" and, with an output bias, "b_o" among them)
    slabs: Callable         # (sizes, dtype) -> {name: Slab}
    run: Callable           # (sizes, eps, w, h, cache, b) -> rows ahead of the output product
    key_views: tuple = ()


def _f32(t: torch.Tensor) -> torch.Tensor:
    return t.float().contiguous()


def _rows(*parts: torch.Tensor) -> torch.Tensor:
    """Row blocks of one product, each padded with zero rows to a multiple of 8 (its columns start on a 16-byte boundary)."""
    return torch.cat([F.pad(t, (0, 0, 0, pad8(t.shape[0]) - t.shape[0])) for t in parts]).contiguous()


# --------------------------------------------------------------------------------------------
# attention with rotated values
# --------------------------------------------------------------------------------------------
def turn_widths(m: dict, dtype: torch.dtype) -> tuple[int, int]:
    """(key width, value width) in the cache: what the bf16 kernels take (zeros behind the sizes), else exact."""
    d, v = m["dim"], m["vdim"]
    if dtype != torch.bfloat16 or d > 192 or v > 128:
        return d, v
    return (64 if d <= 64 else 128 if d <= 128 else 192), (64 if v <= 64 and d <= 128 else 128)


def _turn_fits(m: dict) -> bool:
    return (m["heads"] >= 1 and m["heads"] % m["kv_heads"] == 0 and 1 <= m["dim"] <= 256 and 2 <= m["vdim"] <= 512 and m["vdim"] % 2 == 0
            and m["rot_dim"] % 2 == 0 and 0 <= m["rot_dim"] <= m["dim"])


def _turn_sizes(m: dict) -> tuple[int, int]:
    """Columns of [queries | keys | values] and of the gate."""
    return (m["heads"] + m["kv_heads"]) * m["dim"] + m["kv_heads"] * m["vdim"], m["heads"] * m["vdim"]


def _turn_specs(m: dict, width: int) -> list:
    qkv, hv = _turn_sizes(m)
    return [("w_in", (qkv + hv, width)), ("b_qkv", (qkv,)), ("sink", (m["heads"],)), ("wo", (width, hv)), ("b_o", (width,))]


def _turn_in(m: dict, w: dict) -> list:
    qkv, _ = _turn_sizes(m)
    return [w["w_in"][:qkv], w["w_in"][qkv:]]


def _turn_prepare(m: dict, w: dict, dtype: torch.dtype, is_cuda: bool) -> dict:
    device = w["wo"].device
    return {"w_in": _rows(*_turn_in(m, w)).to(dtype), "wo": w["wo"].to(dtype).contiguous(), **_turn_vectors(m, w, device), "b_o": _f32(w["b_o"])}


def _turn_vectors(m: dict, w: dict, device) -> dict:
    return {"b_qkv": _f32(w["b_qkv"]), "sink": _f32(w["sink"]), "freq": M.rope_frequencies(m["rot_dim"], m["rot_base"], device),
            "vfreq": M.rope_frequencies(m["vdim"], m["rot_base"], device)}


def _turn_slabs(m: dict, dtype: torch.dtype) -> dict:
    kw, vw = turn_widths(m, dtype)
    return {"k_pool": Slab((m["kv_heads"], kw), paged=True), "v_pool": Slab((m["kv_heads"], vw), paged=True)}


def _turn_core(m: dict, eps: float, w: dict, p: torch.Tensor, gate: torch.Tensor, cache: dict, b: M.SpanBatch, scale_out: float, out: torch.Tensor) -> None:
    """out [T, heads * vdim] = scale_out * sigmoid(gate) * (attention turned back)."""
    kp, vp, t, scale = cache["k_pool"], cache["v_pool"], b.tokens, float(m["scale"])
    kw, vw = kp.shape[3], vp.shape[3]
    tl = b.t_long if p.is_cuda and p.dtype == torch.bfloat16 and M.sink_varlen_ok(kw, vw) else 0       # tokens served by the packed kernel
    q, kv = M.turn_prep(p, w["b_qkv"], m["heads"], m["dim"], m["vdim"], w["freq"], w["vfreq"], kp, vp, b, eps, tl > 0 and b.gather is None)
    parts = []
    if tl:
        if b.gather is None:
            k, v, cu_k = kv[0][:tl], kv[1][:tl], b.cu[:b.n_long + 1]
        else:
            rows, cu_k = b.gather[0, 0]
            k, v = M.gather_keys(kp, vp, rows)
        parts.append(M.sink_attention_varlen(q[:tl], k, v, b.cu[:b.n_long + 1], cu_k, scale, w["sink"]))
    if tl < t:
        lo = b.n_long if tl else 0
        seq_of = None if b.seq_of is None or tl else b.seq_of[tl:]
        parts.append(M.sink_attention(q[tl:], kp, vp, b.table[lo:], seq_of, b.kv_len[tl:], scale, w["sink"], b.max_len))
    o = parts[0] if len(parts) == 1 else torch.cat(parts)
    M.turn_back(o, gate, w["vfreq"], b.pos, scale_out, out)


def _turn(m: dict, eps: float, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    qkv, hv = _turn_sizes(m)
    p = ops.linear(h, w["w_in"])
    out = torch.empty(b.tokens, hv, device=h.device, dtype=h.dtype)
    _turn_core(m, eps, w, p[:, :qkv], p[:, pad8(qkv):pad8(qkv) + hv], cache, b, 1.0, out)
    return out


# --------------------------------------------------------------------------------------------
# linear attention with a constant decay
# --------------------------------------------------------------------------------------------
def _decay_fits(m: dict) -> bool:
    return (m["heads"] >= 1 and 1 <= m["dim"] <= 512 and m["vdim"] >= 1 and len(m["decay"]) == m["heads"] and all(0 <= x <= 1 for x in m["decay"]))


def _decay_sizes(m: dict) -> tuple[int, int]:
    """Columns of [queries | keys | values] and of the gate."""
    return m["heads"] * (2 * m["dim"] + m["vdim"]), m["heads"] * m["vdim"]


def _decay_specs(m: dict, width: int) -> list:
    qkv, hv = _decay_sizes(m)
    return [("w_in", (qkv + hv, width)), ("gn", (hv,)), ("wo", (width, hv))]


def _decay_in(m: dict, w: dict) -> list:
    """(gate rows, activated rows) of the input product."""
    qkv, _ = _decay_sizes(m)
    return [w["w_in"][qkv:], w["w_in"][:qkv]]


def _decay_vectors(m: dict, w: dict, scale_out: float = 1.0) -> dict:
    log = [math.log(x) if x > 1e-30 else -80.0 for x in m["decay"]]          # (a decay of zero forgets to below the last bit)
    return {"log_decay": torch.tensor(log, dtype=torch.float32, device=w["wo"].device), "gn": _f32(w["gn"]) * scale_out}


def _decay_prepare(m: dict, w: dict, dtype: torch.dtype, is_cuda: bool) -> dict:
    return {"w_in": _rows(*_decay_in(m, w)).to(dtype), "wo": w["wo"].to(dtype).contiguous(), **_decay_vectors(m, w)}


def _decay_slabs(m: dict, dtype: torch.dtype) -> dict:
    return {"S": Slab((m["heads"], m["dim"], m["vdim"]), fp32=True)}


def _decay_core(m: dict, eps: float, w: dict, qkv: torch.Tensor, gate: torch.Tensor, raw: bool, cache: dict, b: M.SpanBatch, out: torch.Tensor | None) -> torch.Tensor:
    """raw: the rows are not activated yet (the one-token kernel does it)."""
    hd = m["heads"] * m["dim"]
    o = M.scan(M.DECAY, qkv[:, :hd], qkv[:, hd:2 * hd], qkv[:, 2 * hd:2 * hd + m["heads"] * m["vdim"]], M.Gates(a_log=w["log_decay"], raw=raw), 1.0, cache, b)
    return M.gated_norm(o, gate, w["gn"], 1, eps, M.SIGMOID_LAST, out)


def _split_product(h: torch.Tensor, w_in: torch.Tensor, at: int, qkv: int, b: M.SpanBatch) -> tuple[torch.Tensor, torch.Tensor, bool]:
    """(plain columns, columns [at, at + qkv), whether those are not silu-activated yet): one product for single tokens, two — the second with
    the activation in its epilogue — else."""
    if h.is_cuda and b.seq_of is None:
        p = ops.linear(h, w_in)
        return p[:, :at], p[:, at:at + qkv], True
    return ops.linear(h, w_in[:at]), M.linear_silu(h, w_in[at:])[:, :qkv], False


def _decay(m: dict, eps: float, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    qkv, hv = _decay_sizes(m)
    p, x, raw = _split_product(h, w["w_in"], pad8(hv), qkv, b)
    return _decay_core(m, eps, w, x, p[:, :hv], raw, cache, b, None)


# --------------------------------------------------------------------------------------------
# gated linear attention
# --------------------------------------------------------------------------------------------
def _gla_fits(m: dict) -> bool:
    return m["heads"] >= 1 and 1 <= m["dim"] <= 512 and m["vdim"] >= 1 and m["rank"] >= 1 and m["tau"] > 0


def _gla_specs(m: dict, width: int) -> list:         # [q | k | v | gate | decay rank]
    hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
    return [("w_in", (2 * hd + 2 * hv + m["rank"], width)), ("w_a", (hd, m["rank"])), ("b_a", (hd,)), ("gn", (m["vdim"],)), ("wo", (width, hv))]


def _gla_blocks(m: dict) -> list:
    hd, hv = m["heads"] * m["dim"], m["heads"] * m["vdim"]
    return [hd, hd, hv, hv, m["rank"]]


def _gla_prepare(m: dict, w: dict, dtype: torch.dtype, is_cuda: bool) -> dict:
    r = m["rank"]
    return {"w_in": _rows(*w["w_in"].split(_gla_blocks(m))).to(dtype), "w_a": F.pad(w["w_a"], (0, pad8(r) - r)).to(dtype).contiguous(), "b_a": _f32(w["b_a"]),
            "gn": w["gn"].float().repeat(m["heads"]), "wo": w["wo"].to(dtype).contiguous()}


def _gla_slabs(m: dict, dtype: torch.dtype) -> dict:
    return {"S": Slab((m["heads"], m["dim"], m["vdim"]), fp32=True)}


def _gla(m: dict, eps: float, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    p = ops.linear(h, w["w_in"])
    at, cols = 0, []
    for n in _gla_blocks(m):
        cols.append(p[:, at:at + n])
        at += pad8(n)
    z = M.linear_f32(p[:, at - pad8(m["rank"]):at], w["w_a"])
    o = M.scan(M.GLA, cols[0], cols[1], cols[2], M.Gates(z, b0=w["b_a"], cap=float(m["tau"])), m["dim"] ** -0.5, cache, b)
    return M.gated_norm(o, cols[3], w["gn"], m["heads"], eps, M.SILU_LAST)


# --------------------------------------------------------------------------------------------
# selective scan
# --------------------------------------------------------------------------------------------
def _selective_fits(m: dict) -> bool:
    return m["inner"] >= 1 and 1 <= m["state"] <= 512 and m["dt_rank"] >= 1 and m["conv"] >= 1


def _selective_specs(m: dict, width: int) -> list:
    i, n, r = m["inner"], m["state"], m["dt_rank"]
    return [("w_in", (2 * i, width)), ("conv_w", (i, m["conv"])), ("conv_b", (i,)), ("w_x", (r + 2 * n, i)), ("w_dt", (i, r)), ("dt_bias", (i,)), ("a_log", (i, n)),
            ("d_skip", (i,)), ("wo", (width, i))]


def _selective_prepare(m: dict, w: dict, dtype: torch.dtype, is_cuda: bool) -> dict:
    r, n = m["dt_rank"], m["state"]
    return {"w_in": _rows(*w["w_in"].chunk(2)).to(dtype), "conv_w": w["conv_w"].float().t().contiguous(), "conv_b": _f32(w["conv_b"]),
            "w_x": _rows(*w["w_x"].split([r, n, n])).to(dtype), "w_dt": F.pad(w["w_dt"], (0, pad8(r) - r)).to(dtype).contiguous(), "dt_bias": _f32(w["dt_bias"]),
            "a_neg": -torch.exp(w["a_log"].float()).contiguous(), "d_skip": _f32(w["d_skip"]), "wo": w["wo"].to(dtype).contiguous()}


def _selective_slabs(m: dict, dtype: torch.dtype) -> dict:
    return {"S": Slab((m["inner"], m["state"]), fp32=True), "conv": Slab((m["conv"] - 1, m["inner"]))}


def _selective(m: dict, eps: float, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    i, n, r = m["inner"], m["state"], pad8(m["dt_rank"])
    p = ops.linear(h, w["w_in"])
    x = M.conv_silu(p[:, :i], w["conv_w"], w["conv_b"], cache["conv"], b)
    px = ops.linear(x, w["w_x"])
    dt = M.linear_f32(px[:, :r], w["w_dt"])
    return M.selective_scan(x, dt, px[:, r:r + n], px[:, r + pad8(n):r + pad8(n) + n], p[:, pad8(i):pad8(i) + i], w["dt_bias"], w["a_neg"], w["d_skip"], cache["S"], b)


# --------------------------------------------------------------------------------------------
# two mixers side by side
# --------------------------------------------------------------------------------------------
PAIRABLE = ("turn", "decay")        # (left, right): attention beside a recurrence


def _pair_fits(m: dict) -> bool:
    return (m["left"]["kind"], m["right"]["kind"]) == PAIRABLE and _turn_fits(m["left"]) and _decay_fits(m["right"])


def _pair_specs(m: dict, width: int) -> list:
    return [(f"{s}.{n}", shp) for s in ("left", "right") for n, shp in KINDS[m[s]["kind"]].specs(m[s], width)]


def _of(side: str, d: dict) -> dict:
    return {k[len(side) + 1:]: t for k, t in d.items() if k.startswith(side + ".")}


def _pair_prepare(m: dict, w: dict, dtype: torch.dtype, is_cuda: bool) -> dict:
    lw, rw = _of("left", w), _of("right", w)
    out = {"w_in": _rows(*_turn_in(m["left"], lw), *_decay_in(m["right"], rw)).to(dtype), "wo": torch.cat([lw["wo"], rw["wo"]], 1).to(dtype).contiguous(),
           "b_o": _f32(lw["b_o"]) * m["left_scale"]}
    out.update({f"left.{k}": t for k, t in _turn_vectors(m["left"], lw, lw["wo"].device).items()})
    out.update({f"right.{k}": t for k, t in _decay_vectors(m["right"], rw, m["right_scale"]).items()})
    return out


def _pair_slabs(m: dict, dtype: torch.dtype) -> dict:
    return {f"{s}.{n}": x for s in ("left", "right") for n, x in KINDS[m[s]["kind"]].slabs(m[s], dtype).items()}


def _pair(m: dict, eps: float, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    (lq, lv), (rq, rv) = _turn_sizes(m["left"]), _decay_sizes(m["right"])
    g0 = pad8(lq)
    r0 = g0 + pad8(lv)
    p, x, raw = _split_product(h, w["w_in"], r0 + pad8(rv), rq, b)
    out = torch.empty(b.tokens, lv + rv, device=h.device, dtype=h.dtype)
    with M.beside(h, b) as side:            # in single-token steps the two halves are chains of small kernels
        with side():
            _decay_core(m["right"], eps, _of("right", w), x, p[:, r0:r0 + rv], raw, _of("right", cache), b, out[:, lv:])
        _turn_core(m["left"], eps, _of("left", w), p[:, :lq], p[:, g0:g0 + lv], _of("left", cache), b, float(m["left_scale"]), out[:, :lv])
    return out


KINDS = {
    "turn": Kind(_turn_fits, _turn_specs, _turn_prepare, _turn_slabs, _turn, ((0, 0),)),
    "decay": Kind(_decay_fits, _decay_specs, _decay_prepare, _decay_slabs, _decay),
    "gla": Kind(_gla_fits, _gla_specs, _gla_prepare, _gla_slabs, _gla),
    "selective": Kind(_selective_fits, _selective_specs, _selective_prepare, _selective_slabs, _selective),
    "pair": Kind(_pair_fits, _pair_specs, _pair_prepare, _pair_slabs, _pair, ((0, 0),)),
}
