"""Mixer stacks: decoder-only models whose layers each choose their own sequence mixer, served by the rollout engine.

A layer is  x <- x + norm1(mixer(pre1(x))),  x <- x + norm2(ff(pre2(x)))  over an fp32 residual stream: RMS norms on the sublayer outputs
and, with ``ModelConfig.sandwich_norm``, on their inputs too; ``norm_offset`` is added to the stored weights of these norms and of the
final one.

With ``ModelConfig.parallel_block`` a layer is  h = pre1(x),  X' = x + ls1 mixer(h + conv1(h)) + ls2 ff(h + conv2(h)): one norm (with
``layer_norm`` around the mean), short causal convolutions over time on what either sublayer reads (``input_conv`` taps, carried in
the state slots), element-wise scales on their results (``layer_scale``).  With ``depth_average`` the next layer reads a learned average
x = sum_j depth[j] X_j over the embedding output X_0 and the results X_j of the layers so far; they are kept in fp32 for the step's
tokens, and x itself is never stored: the kernel that adds a layer's results recomputes it from them.

With ``ModelConfig.streams`` the residual is that many streams X_s (hyper-connections), all the embedding output at first, and every
sublayer q has maps of its own:  u = sum_s in_q[s] X_s,  y = sublayer(norm_q(u)),  X_t <- sum_s mix_q[s, t] X_s + out_q[t] y.  Norms are on
the inputs; the model's output is the sum of the streams.  ``scalar_norm``: the weight of such a norm is one number.  One kernel ends a
sublayer and begins the next: it reads and writes the streams once.

Mixers (``LAYER_KINDS``):
  ``ssd``     Mamba-2 state-space duality: causal convolution, scalar-decay recurrence, gate before a grouped norm
  ``mlstm``   xLSTM matrix memory with exponential gates
  ``delta``   gated delta rule: short convolutions, unit queries and keys, one decay per head, gated norm per head
  ``latent``  multi-head latent attention with query bottleneck, rotary key part and a softmax sink
  ``window``  grouped-query attention in a sliding window with kept first tokens; queries and keys are normed over the whole projection
              and partly rotated in neighbouring pairs, the values are the keys as projected
  ``diff``    differential attention in a sliding window: two softmax maps per head over the same values, a1 - lambda a2, normed per head;
              projection biases, queries and keys normed per head and map, rotate-half positions with Llama 3.1 frequency scaling
  and those of ``mixer_kinds.py``
Feed-forwards (``act``): ``gelu``, ``clamped_glu``, ``poly`` (up, a N(z) + b N(z^2) + c N(z^3) + e with RMS norms N, down) or ``moe`` (gated
experts and a shared one; ``router``: ``sigmoid_in``, the ``top`` largest sigmoid scores weigh the experts' inputs, or ``softmax``, the ``top`` largest
softmax scores over their sum weigh the outputs; with ``limit`` and ``alpha`` the experts are clamped, ``shared_limit`` being the shared one's).  A layer
may reuse the weights of an earlier one (``weights_of``) while keeping a cache or state of its own.

``ModelConfig.layers`` holds one plain dict per layer: {"kind", "sizes", "ff" (0: no feed-forward), "weights_of" (own index when the
layer owns its weights)} and what its feed-forward needs ("act", "limit", "alpha", "experts", "top", "shared", "router", "shared_limit").  ``stacks.py`` reads the designs' config.json and
checkpoint names; another design built from the same mixers needs only another reader and name map.

Everything is one function of a packed step (ops/mixers.py ``SpanBatch``): prompts, portions of prompts and decoded tokens take the
same path, and the kernels pick chunked or token-by-token work by span length.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from .. import ops
from ..ops import mixers as M
from ..ops import reference as ref
from .config import ModelConfig
from .mixer_kinds import KINDS

LAYER_KINDS = ("ssd", "mlstm", "delta", "latent", "window", "diff", *KINDS)
MAPS = 2                            # softmax maps of a differential attention head
MAX_EXPERTS = 1024
MAX_STREAMS = 16
ROUTERS = ("sigmoid_in", "softmax")


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


def owner(cfg: ModelConfig, i: int) -> int:
    """Index of the layer whose weights layer ``i`` uses."""
    seen = set()
    while cfg.layers[i]["weights_of"] != i:
        if i in seen:
            raise ValueError("weights_of forms a cycle")
        seen.add(i)
        i = cfg.layers[i]["weights_of"]
    return i


def validate(cfg: ModelConfig) -> None:
    if len(cfg.layers) != cfg.num_layers or not cfg.layers:
        raise ValueError("a mixer stack needs one entry of ``layers`` per layer")
    if cfg.parallel_block and (cfg.sandwich_norm or cfg.input_conv < 0):
        raise ValueError("parallel blocks have one norm, on the input")
    if not cfg.parallel_block and (cfg.layer_norm or cfg.input_conv or cfg.layer_scale or cfg.depth_average):
        raise ValueError("layer norms, input convolutions, layer scales and depth averages need parallel blocks")
    if cfg.streams and (not 1 <= cfg.streams <= MAX_STREAMS or cfg.parallel_block or cfg.sandwich_norm):
        raise ValueError(f"residual streams: 1 to {MAX_STREAMS}, and norms on the sublayers' inputs only")
    if cfg.scalar_norm and not cfg.streams:
        raise ValueError("norms with one number as their weight need residual streams")
    for i, lay in enumerate(cfg.layers):
        kind, m = lay["kind"], lay["sizes"]
        if kind not in LAYER_KINDS:
            raise ValueError(f"layer {i}: unknown mixer {kind!r}")
        if not 0 <= lay["weights_of"] < cfg.num_layers:
            raise ValueError(f"layer {i}: weights_of is not a layer")
        j = owner(cfg, i)
        if {k: v for k, v in cfg.layers[j].items() if k != "weights_of"} != {k: v for k, v in lay.items() if k != "weights_of"}:
            raise ValueError(f"layer {i} differs from layer {j} whose weights it uses")
        if kind in KINDS and not KINDS[kind].fits(m):
            raise ValueError(f"layer {i}: {kind} sizes")
        if kind == "ssd" and (m["heads"] % m["groups"] or (m["heads"] * m["vdim"]) % m["norm_groups"] or m["conv"] < 1 or m["state"] > 512):
            raise ValueError(f"layer {i}: ssd sizes")
        if kind == "mlstm" and (m["dim"] > 512 or m["gate_cap"] <= 0):
            raise ValueError(f"layer {i}: mlstm sizes")
        if kind == "latent" and (m["rot_dim"] % 2 or m["rot_dim"] > 512 or m["kv_rank"] > 1024):
            raise ValueError(f"layer {i}: latent sizes")
        if cfg.depth_average and j != i:
            raise ValueError(f"layer {i}: a depth average has its own length in every layer")
        if kind in ("delta", "window", "diff") and m["heads"] % m["kv_heads"]:
            raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
        if kind == "delta" and (m["dim"] > 512 or m["conv"] < 1):
            raise ValueError(f"layer {i}: delta sizes")
        if kind == "window" and (m["vdim"] != m["dim"] or m["rot_dim"] % 2 or not 0 <= m["rot_dim"] <= min(512, m["dim"]) or m["dim"] > 1024 or m["window"] < 1
                                 or m["keep_first"] < 0):
            raise ValueError(f"layer {i}: window sizes (values are keys: vdim equals dim)")
        if kind == "diff" and (m["rot_dim"] % 2 or not 0 <= m["rot_dim"] <= min(512, m["dim"]) or not 1 <= m["dim"] <= 256 or not 1 <= m["vdim"] <= 512
                               or m["window"] < 1):
            raise ValueError(f"layer {i}: diff sizes")
        if lay["ff"] and lay.get("act", "gelu") not in ("gelu", "clamped_glu", "poly", "moe"):
            raise ValueError(f"layer {i}: unknown feed-forward {lay['act']!r}")
        if lay["ff"] and lay.get("act") == "moe" and not (1 <= lay["top"] <= lay["experts"] <= MAX_EXPERTS and lay["shared"] >= 0
                                                              and (cfg.parallel_block or cfg.streams) and lay.get("router", ROUTERS[0]) in ROUTERS):
            raise ValueError(f"layer {i}: experts (parallel blocks and residual streams only)")


# --------------------------------------------------------------------------------------------
# parameters (our names; weights of a layer that reuses another's exist once)
# --------------------------------------------------------------------------------------------
def layer_param_specs(cfg: ModelConfig, i: int) -> list[tuple[str, tuple[int, ...]]]:
    lay, w = cfg.layers[i], cfg.hidden_size
    m, h, v = lay["sizes"], lay["sizes"].get("heads"), lay["sizes"].get("vdim")
    out: list[tuple[str, tuple[int, ...]]]
    if cfg.streams:
        out, n = [], cfg.streams
        for q in ("1", "2") if lay["ff"] else ("1",):
            out += [("pre" + q, () if cfg.scalar_norm else (w,)), (f"hc{q}.in", (n,)), (f"hc{q}.out", (n,)), (f"hc{q}.mix", (n, n))]
    elif cfg.parallel_block:
        out = [("pre1", (w,))]
        for n in ("1", "2") if lay["ff"] else ("1",):
            out += ([("ls" + n, (w,))] if cfg.layer_scale else []) + ([("conv" + n, (w, cfg.input_conv))] if cfg.input_conv else [])
        out += [("depth", (i + 2,))] if cfg.depth_average else []
    else:
        out = ([("pre1", (w,))] if cfg.sandwich_norm else []) + [("norm1", (w,))]
    if lay["kind"] in KINDS:
        out += KINDS[lay["kind"]].specs(m, w)
    elif lay["kind"] == "ssd":          # one projection [gate | x | B | C]; the step sizes keep their own fp32-accumulated one
        ch = h * v + 2 * m["groups"] * m["state"]
        out += [("w_in", (h * v + ch, w)), ("w_dt", (h, w)), ("conv_w", (ch, m["conv"])), ("conv_b", (ch,)), ("dt_bias", (h,)), ("a_log", (h,)),
                ("d_skip", (h,)), ("gn", (h * v,)), ("wo", (w, h * v))]
    elif lay["kind"] == "mlstm":        # [q | k | v | output gate] and [input gate | forget gate]
        out += [("w_in", (2 * h * m["dim"] + 2 * h * v, w)), ("w_if", (2 * h, w)), ("b_if", (2 * h,)), ("gn", (h * v,)), ("wo", (w, h * v))]
    elif lay["kind"] == "delta":        # [q | k | v | output gate], [decay | write strength]; the convolution runs over [q | k | v]
        qk = m["kv_heads"] * m["dim"]
        out += [("w_in", (2 * qk + 2 * h * v, w)), ("w_ab", (2 * h, w)), ("conv_w", (2 * qk + h * v, m["conv"])), ("dt_bias", (h,)), ("a_log", (h,)),
                ("gn", (v,)), ("wo", (w, h * v))]
    elif lay["kind"] == "window":       # [q | k]
        hd, gd = h * m["dim"], m["kv_heads"] * m["dim"]
        out += [("wqk", (hd + gd, w)), ("q_norm", (hd,)), ("k_norm", (gd,)), ("wo", (w, hd))]
    elif lay["kind"] == "diff":         # [q | k | v], q and k head by head as [map 1 | map 2]; map_mix: four vectors that make lambda
        rows = MAPS * (h + m["kv_heads"]) * m["dim"] + m["kv_heads"] * v
        out += [("wqkv", (rows, w)), ("b_qkv", (rows,)), ("q_norm", (m["dim"],)), ("k_norm", (m["dim"],)), ("map_mix", (4 * m["dim"],)), ("wo", (w, h * v))]
    else:                               # [query latent | key-value latent | shared rotary key]
        r, qr, d, rd = m["kv_rank"], m["q_rank"], m["dim"], m["rot_dim"]
        out += [("wa", (qr + r + rd, w)), ("q_ln", (qr,)), ("kv_ln", (r,)), ("wq_up", (h * (d + rd), qr)), ("wk_up", (h * d, r)), ("wv_up", (h * v, r)),
                ("sink", (h,)), ("wo", (w, h * v))]
    if lay["ff"]:
        f, act = lay["ff"], lay.get("act", "gelu")
        if not cfg.parallel_block and not cfg.streams:
            out += ([("pre2", (w,))] if cfg.sandwich_norm else []) + [("norm2", (w,))]
        # gate and up rows: interleaved in blocks of 128 (as the llama family's) where ff allows it, else one after the other
        if act == "moe":                # experts one after the other
            n, fs = lay["experts"], lay["shared"]
            out += [("router", (n, w)), ("ewgu", (n * 2 * f, w)), ("ewd", (n * w, f))] + ([("swgu", (2 * fs, w)), ("swd", (w, fs))] if fs else [])
        else:
            out += [("wgu", (2 * f, w)) if act == "clamped_glu" else ("wup", (f, w)), ("wdown", (w, f))] + ([("act", (4,))] if act == "poly" else [])
    return out


def gate_up_stacks(lay: dict) -> list[tuple[str, int, int]]:
    """(name, how many, width) of a layer's stacks of gate and up rows."""
    if not lay["ff"] or lay.get("act") not in ("clamped_glu", "moe"):
        return []
    if lay["act"] == "clamped_glu":
        return [("wgu", 1, lay["ff"])]
    return [("ewgu", lay["experts"], lay["ff"])] + ([("swgu", 1, lay["shared"])] if lay["shared"] else [])


def num_params(cfg: ModelConfig) -> int:
    n = 2 * cfg.vocab_size * cfg.hidden_size + (1 if cfg.scalar_norm else cfg.hidden_size)
    for i in range(cfg.num_layers):
        if owner(cfg, i) == i:
            for _, shp in layer_param_specs(cfg, i):
                k = 1
                for s in shp:
                    k *= s
                n += k
    return n


def init_param_(name: str, t: torch.Tensor, cfg: ModelConfig, generator=None) -> bool:
    """Random init of the tensors the generic rules do not cover; False when they do."""
    base = name.split(".")[-1]
    if base in ("pre1", "norm1", "pre2", "norm2", "norm_w"):
        t.fill_(1.0 - cfg.norm_offset)
    elif base in ("in", "out"):     # streams: read their mean, write to all of them
        t.fill_(1.0 if base == "out" else 1.0 / cfg.streams)
    elif base == "mix":
        t.copy_(torch.eye(cfg.streams))
    elif base in ("gn", "q_ln", "kv_ln", "q_norm", "k_norm", "d_skip", "ls1", "ls2"):
        t.fill_(1.0)
    elif base in ("conv_b", "sink", "b_qkv", "map_mix", "b_o"):
        t.zero_()
    elif base == "depth":           # the layer's own result
        t.zero_()
        t[-1] = 1.0
    elif base == "act":
        t.copy_(torch.tensor([1 / 3, 1 / 3, 1 / 3, 0.0]))
    elif base in ("conv1", "conv2"):
        t.normal_(0.0, 0.1 * t.shape[1] ** -0.5, generator=generator)
    elif base == "b_a":             # slow decays
        t.fill_(3.0)
    elif base == "a_log" and t.dim() == 2:
        t.copy_(torch.log(torch.arange(1, t.shape[1] + 1, device=t.device, dtype=torch.float32)).expand(t.shape))
    elif base == "a_log":
        t.copy_(torch.linspace(-2.0, 1.0, t.numel(), device=t.device))
    elif base == "dt_bias":
        t.fill_(-2.0)
    elif base == "b_if":
        t.zero_()
        t[t.numel() // 2:] = 3.0
    elif base == "conv_w":
        t.normal_(0.0, t.shape[1] ** -0.5, generator=generator)
    elif base in ("w_in", "w_dt", "w_if", "wa", "wq_up", "wk_up", "wv_up", "wo", "wup", "wdown", "w_ab", "wqk", "wgu", "wqkv", "router", "ewgu", "ewd",
                  "swgu", "swd", "w_a", "w_x"):
        t.normal_(0.0, t.shape[1] ** -0.5, generator=generator)
    else:
        return False
    return True


# --------------------------------------------------------------------------------------------
# run-time weights
# --------------------------------------------------------------------------------------------
_STREAM_NORMS = ("pre1", "norm1", "pre2", "norm2")               # of the residual stream: ``norm_offset`` applies
_VECTORS = ("gn", "q_ln", "kv_ln", "q_norm", "k_norm", "conv_b", "dt_bias", "a_log", "d_skip", "b_if", "sink", "b_qkv", "ls1", "ls2", "depth", "act")
_DERIVED_ONLY = ("wq_up", "wk_up", "wv_up", "map_mix")              # stored tensors that only enter others


def packs(m: dict, dtype: torch.dtype, is_cuda: bool) -> bool:
    """Long spans of this ``window`` or ``diff`` layer run on the packed tcgen05 attention."""
    return is_cuda and dtype == torch.bfloat16 and max(m["dim"], m.get("vdim", 0)) <= 128


def cache_width(m: dict, dtype: torch.dtype) -> int:
    """Width of a cached key of a ``window`` layer: what the bf16 kernels take (64 or 128, zeros behind the key), else its own."""
    return m["dim"] if dtype != torch.bfloat16 or m["dim"] > 128 else (64 if m["dim"] <= 64 else 128)


def map_widths(m: dict, dtype: torch.dtype) -> tuple[int, int]:
    """(key width of one map, value width) of a ``diff`` layer in the cache: what the bf16 kernels take (zeros behind the sizes), else exact."""
    if dtype != torch.bfloat16 or max(m["dim"], m["vdim"]) > 128:
        return m["dim"], m["vdim"]
    return next(x for x in (32, 64, 128) if m["dim"] <= x), 64 if m["vdim"] <= 64 else 128


def query_width(m: dict, dtype: torch.dtype, is_cuda: bool) -> int:
    """Per-head query width at run time: padded to what the packed attention kernel takes (128 or 192), or exact when that kernel cannot
    serve the sizes (fp32, wider heads)."""
    d = m["dim"] + m["rot_dim"]
    return d if not expands(m, dtype, is_cuda) else (128 if d <= 128 else 192)


def expands(m: dict, dtype: torch.dtype, is_cuda: bool) -> bool:
    """Long spans of this layer run on expanded keys and values (packed tcgen05 attention) instead of the absorbed form."""
    return is_cuda and dtype == torch.bfloat16 and m["vdim"] <= 128 and m["dim"] + m["rot_dim"] <= 192 and (m["kv_rank"] + m["rot_dim"]) % 8 == 0


def _pad_heads(w: torch.Tensor, heads: int, rows: int) -> torch.Tensor:
    """[heads * n, in] -> [heads * rows, in], zero rows behind every head's own."""
    t = w.reshape(heads, -1, w.shape[-1])
    return F.pad(t, (0, 0, 0, rows - t.shape[1])).reshape(heads * rows, -1)


def prepare_layer(cfg: ModelConfig, i: int, w: dict, dtype: torch.dtype, old: dict | None = None) -> dict:
    """Weights of layer ``i`` in run-time form: vectors in fp32, matrices in ``dtype`` with the layouts the kernels want.  ``old`` (the
    previous result) is overwritten in place where shapes agree, so captured graphs stay valid across weight updates."""
    lay = cfg.layers[i]
    m, h = lay["sizes"], lay["sizes"].get("heads")
    own = {} if lay["kind"] not in KINDS else {n for n, _ in KINDS[lay["kind"]].specs(m, cfg.hidden_size)}
    device = next(iter(w.values())).device
    is_cuda = device.type == "cuda"
    out: dict[str, torch.Tensor] = {}
    if own:
        out.update(KINDS[lay["kind"]].prepare(m, w, dtype, is_cuda))
    for k, t in w.items():
        if k in own:
            continue
        if k.startswith("hc"):
            out[k] = t.float().contiguous()
        elif k in _STREAM_NORMS:
            out[k] = (t.float() + cfg.norm_offset).reshape(-1).contiguous() if cfg.norm_offset else t.float().reshape(-1).contiguous()
        elif k == "gn" and t.numel() < h * m["vdim"]:             # one weight for all heads
            out[k] = t.float().repeat(h)
        elif k in _VECTORS:
            out[k] = t.float().contiguous()
        elif k in ("conv_w", "conv1", "conv2"):
            out[k] = t.float().t().contiguous()                     # [taps, channels]
        elif k not in _DERIVED_ONLY:
            t = t if t.dtype == dtype else t.to(dtype)
            if k in ("w_in", "wqk", "wqkv") and is_cuda and t.shape[0] % 8:
                t = F.pad(t, (0, 0, 0, _pad8(t.shape[0]) - t.shape[0]))
            out[k] = t.contiguous()
    if lay["kind"] == "window":
        out["freq"] = M.rope_frequencies(m["rot_dim"], m["rot_base"], device)
    if lay["kind"] == "diff":
        out["freq"] = M.scaled_frequencies(m["rot_dim"], m["rot_base"], m.get("rot_scaling"), device)
        q1, k1, q2, k2 = w["map_mix"].float().chunk(4)
        out["lam"] = ((q1 * k1).sum().exp() - (q2 * k2).sum().exp() + m["diff"]).reshape(1)
    for name, count, f in gate_up_stacks(lay):
        if is_cuda and dtype == torch.bfloat16 and f % 128:
            # the fused gate / up kernels want 128-row blocks: zero rows behind the last ones
            pad, down = -f % 128, {"wgu": "wdown", "ewgu": "ewd", "swgu": "swd"}[name]
            out[name] = torch.cat([ref.interleave_gate_up(*(F.pad(t, (0, 0, 0, pad)) for t in x.chunk(2))) for x in out[name].chunk(count)])
            out[down] = F.pad(out[down], (0, pad))
    if lay["kind"] == "latent":
        d, rd, v, r = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
        dq = query_width(m, dtype, is_cuda)
        up = {k: w[k].to(dtype) for k in ("wq_up", "wk_up", "wv_up")}
        out["wq"] = _pad_heads(up["wq_up"], h, dq).contiguous()
        out["wk_abs"] = up["wk_up"].reshape(h, d, r).contiguous()                       # folds the key up-projection into a query
        out["wv_abs"] = up["wv_up"].reshape(h, v, r).transpose(1, 2).contiguous()       # folds the value up-projection into an output
        out["freq"] = M.rope_frequencies(rd, m["rot_base"], device)
        if expands(m, dtype, is_cuda):
            # cache row -> every head's [key | rotary key | 0] and [value | 0]: the rotary part is copied by identity rows
            wk = torch.zeros(h, dq, r + rd, dtype=dtype, device=device)
            wk[:, :d, :r] = up["wk_up"].reshape(h, d, r)
            wk[:, d:d + rd, r:] = torch.eye(rd, dtype=dtype, device=wk.device)
            wv = torch.zeros(h, 128, r + rd, dtype=dtype, device=wk.device)
            wv[:, :v, :r] = up["wv_up"].reshape(h, v, r)
            out["w_expand"] = torch.cat([wk.reshape(h * dq, -1), wv.reshape(h * 128, -1)]).contiguous()
    if old is not None:
        for k, t in out.items():
            o = old.get(k)
            derived = k not in w or t.data_ptr() != w[k].data_ptr() or t.shape != w[k].shape
            if derived and o is not None and o.shape == t.shape and o.dtype == t.dtype:
                out[k] = o.copy_(t)
    return out


def prepare(cfg: ModelConfig, layer_w: list[dict], dtype: torch.dtype, old: list[dict] | None = None) -> list[dict]:
    done: dict[int, dict] = {}
    for i in range(cfg.num_layers):
        j = owner(cfg, i)
        if j not in done:
            done[j] = prepare_layer(cfg, j, layer_w[j], dtype, old[j] if old else None)
    return [done[owner(cfg, i)] for i in range(cfg.num_layers)]


def prepare_head(cfg: ModelConfig, head_w: dict, dtype: torch.dtype, old: dict | None = None) -> dict:
    norm = head_w["norm_w"].float().expand(cfg.hidden_size).contiguous()
    if cfg.norm_offset:
        norm = norm + cfg.norm_offset
    if old is not None and norm.data_ptr() != head_w["norm_w"].data_ptr():
        norm = old["norm_w"].copy_(norm)
    return {"norm_w": norm, "lm_head": head_w["lm_head"].to(dtype)}


# --------------------------------------------------------------------------------------------
# caches and states
# --------------------------------------------------------------------------------------------
def cache_bytes(cfg: ModelConfig, dtype: torch.dtype) -> tuple[int, int]:
    """(paged-cache bytes per token, state bytes per slot) of the whole stack."""
    es = torch.empty(0, dtype=dtype).element_size()
    tok = slot = 0
    for lay in cfg.layers:
        m, h, v = lay["sizes"], lay["sizes"].get("heads"), lay["sizes"].get("vdim")
        if lay["kind"] in KINDS:
            for s in KINDS[lay["kind"]].slabs(m, dtype).values():
                tok, slot = (tok + s.bytes(es), slot) if s.paged else (tok, slot + s.bytes(es))
        elif lay["kind"] == "latent":
            tok += (m["kv_rank"] + m["rot_dim"]) * es
        elif lay["kind"] == "window":
            tok += 2 * m["kv_heads"] * cache_width(m, dtype) * es
        elif lay["kind"] == "diff":
            kw, vw = map_widths(m, dtype)
            tok += m["kv_heads"] * (MAPS * kw + vw) * es
        elif lay["kind"] == "delta":
            slot += 4 * h * v * m["dim"] + es * (m["conv"] - 1) * (h * v + 2 * m["kv_heads"] * m["dim"])
        elif lay["kind"] == "ssd":
            slot += 4 * h * v * m["state"] + es * (m["conv"] - 1) * (h * v + 2 * m["groups"] * m["state"])
        else:
            slot += 4 * h * (m["dim"] * v + m["dim"] + 1)
        slot += es * max(0, cfg.input_conv - 1) * cfg.hidden_size
    return tok, slot


def key_views(cfg: ModelConfig) -> list[tuple[int, int]]:
    """The distinct (window, kept first tokens) of the stack's attention layers; (0, 0) sees every key."""
    own = {v for lay in cfg.layers if lay["kind"] in KINDS for v in KINDS[lay["kind"]].key_views}
    return sorted(own | {(lay["sizes"].get("window", 0), lay["sizes"].get("keep_first", 0)) for lay in cfg.layers
                         if lay["kind"] in ("latent", "window", "diff")})


def make_cache(cfg: ModelConfig, i: int, num_blocks: int, num_slots: int, device, dtype: torch.dtype) -> dict[str, torch.Tensor]:
    """Cache of layer ``i``: page pools (attention), state pools (recurrences, convolutions; slot 0 belongs to idle batch rows)."""
    out = _mixer_cache(cfg, i, num_blocks, num_slots, device, dtype)
    if cfg.input_conv:              # the last inputs of both sublayers' convolutions, which are the same rows
        out["input"] = torch.zeros(num_slots, cfg.input_conv - 1, cfg.hidden_size, device=device, dtype=dtype)
    return out


def _mixer_cache(cfg: ModelConfig, i: int, num_blocks: int, num_slots: int, device, dtype: torch.dtype) -> dict[str, torch.Tensor]:
    lay = cfg.layers[i]
    m, h, v = lay["sizes"], lay["sizes"].get("heads"), lay["sizes"].get("vdim")
    if lay["kind"] in KINDS:
        return {n: s.make(num_blocks, num_slots, device, dtype) for n, s in KINDS[lay["kind"]].slabs(m, dtype).items()}
    if lay["kind"] == "latent":
        return {"pool": torch.zeros(num_blocks, 1, M.PAGE, m["kv_rank"] + m["rot_dim"], device=device, dtype=dtype)}
    if lay["kind"] == "window":
        shape = (num_blocks, m["kv_heads"], M.PAGE, cache_width(m, dtype))
        return {n: torch.zeros(shape, device=device, dtype=dtype) for n in ("k_pool", "v_pool")}
    if lay["kind"] == "diff":           # keys [map 1 | map 2]
        kw, vw = map_widths(m, dtype)
        return {n: torch.zeros(num_blocks, m["kv_heads"], M.PAGE, x, device=device, dtype=dtype) for n, x in (("k_pool", MAPS * kw), ("v_pool", vw))}
    f32 = dict(device=device, dtype=torch.float32)
    if lay["kind"] == "delta":
        ch = 2 * m["kv_heads"] * m["dim"] + h * v
        return {"S": torch.zeros(num_slots, h, m["dim"], v, **f32), "conv": torch.zeros(num_slots, m["conv"] - 1, ch, device=device, dtype=dtype)}
    if lay["kind"] == "ssd":
        ch = h * v + 2 * m["groups"] * m["state"]
        return {"S": torch.zeros(num_slots, h, m["state"], v, **f32), "conv": torch.zeros(num_slots, m["conv"] - 1, ch, device=device, dtype=dtype)}
    return {"S": torch.zeros(num_slots, h, m["dim"], v, **f32), "n": torch.zeros(num_slots, h, m["dim"], **f32), "m": torch.zeros(num_slots, h, **f32)}


def copy_cache(cache: dict, src_pages: torch.Tensor, dst_pages: torch.Tensor, src_slots: torch.Tensor, dst_slots: torch.Tensor) -> None:
    """Duplicate pages / state slots of one layer (the members of an n-sample group continue from their donor's prompt)."""
    for k, t in cache.items():
        src, dst = (src_pages, dst_pages) if k.endswith("pool") else (src_slots, dst_slots)
        if src.numel():
            t.index_copy_(0, dst, t.index_select(0, src))


# --------------------------------------------------------------------------------------------
# forward
# --------------------------------------------------------------------------------------------
def _ssd(cfg: ModelConfig, m: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
    p = ops.linear(h, w["w_in"])
    dt = M.linear_f32(h, w["w_dt"])
    z, xbc = p[:, :inner], p[:, inner:2 * inner + 2 * gn]
    xbc = M.conv_silu(xbc, w["conv_w"], w["conv_b"], cache["conv"], b)
    y = M.scan(M.SSD, xbc[:, inner + gn:], xbc[:, inner:inner + gn], xbc[:, :inner],
               M.Gates(dt, b0=w["dt_bias"], a_log=w["a_log"], d_skip=w["d_skip"]), 1.0, cache, b)
    return M.gated_norm(y, z, w["gn"], m["norm_groups"], cfg.rms_norm_eps, M.SILU_FIRST)


def _mlstm(cfg: ModelConfig, m: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    nh = m["heads"]
    hd, hv = nh * m["dim"], nh * m["vdim"]
    p = ops.linear(h, w["w_in"])
    g = M.linear_f32(h, w["w_if"])
    o = M.scan(M.MLSTM, p[:, :hd], p[:, hd:2 * hd], p[:, 2 * hd:2 * hd + hv],
               M.Gates(g[:, :nh], g[:, nh:], w["b_if"][:nh], w["b_if"][nh:], cap=float(m["gate_cap"])), m["dim"] ** -0.5, cache, b)
    return M.gated_norm(o, p[:, 2 * hd + hv:2 * hd + 2 * hv], w["gn"], nh, cfg.rms_norm_eps, M.SIGMOID_LAST)


def _latent(cfg: ModelConfig, m: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    nh, d, rd, v, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    t, pool, scale = b.tokens, cache["pool"], float(m["scale"])
    tl = b.t_long if expands(m, h.dtype, h.is_cuda) else 0          # tokens served on expanded keys
    cq, entry = M.latent_prep(ops.linear(h, w["wa"]), w["q_ln"], w["kv_ln"], w["freq"], pool, b, cfg.rms_norm_eps, tl > 0 and b.gather is None)
    q = ops.linear(cq, w["wq"]).view(t, nh, -1)
    M.rope_(q, d, w["freq"], b.pos)
    out = []
    if tl:
        if b.gather is None:
            src, cu_k = entry[:tl], b.cu[:b.n_long + 1]
        else:
            rows, cu_k = b.gather[0, 0]
            src = pool.view(-1, r + rd).index_select(0, rows)
        kv = ops.linear(src, w["w_expand"])
        dq = q.shape[-1]
        k, vv = kv[:, :nh * dq].view(-1, nh, dq), kv[:, nh * dq:].view(-1, nh, 128)
        a = M.sink_attention_varlen(q[:tl], k, vv, b.cu[:b.n_long + 1], cu_k, scale, w["sink"])
        out.append(a[..., :v].reshape(tl, nh * v))
    if tl < t:
        qs = q[tl:]
        q_lat = torch.bmm(qs[..., :d].transpose(0, 1), w["wk_abs"])
        lo = b.n_long if tl else 0
        seq_of = None if b.seq_of is None or tl else b.seq_of[tl:]
        o_lat = M.latent_attention(q_lat, qs, d, pool, b.table[lo:], seq_of, b.kv_len[tl:], w["sink"], scale, b.max_len)
        out.append(torch.bmm(o_lat, w["wv_abs"]).transpose(0, 1).reshape(t - tl, nh * v))
    return out[0] if len(out) == 1 else torch.cat(out)


def _delta(cfg: ModelConfig, m: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    nh, qk = m["heads"], m["kv_heads"] * m["dim"]
    hv = nh * m["vdim"]
    p = ops.linear(h, w["w_in"])
    ab = M.linear_f32(h, w["w_ab"])
    c = M.conv_silu(p[:, :2 * qk + hv], w["conv_w"], None, cache["conv"], b)
    o = M.scan(M.DELTA, c[:, :qk], c[:, qk:2 * qk], c[:, 2 * qk:], M.Gates(ab[:, :nh], ab[:, nh:], b0=w["dt_bias"], a_log=w["a_log"]), m["dim"] ** -0.5,
               cache, b)
    return M.gated_norm(o, p[:, 2 * qk + hv:2 * qk + 2 * hv], w["gn"], nh, cfg.rms_norm_eps, M.SILU_LAST)


def _window(cfg: ModelConfig, m: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    nh, d, t = m["heads"], m["dim"], b.tokens
    view = (m["window"], m["keep_first"])
    scale, kp, vp = float(m["scale"]), cache["k_pool"], cache["v_pool"]
    tl = b.t_long if packs(m, h.dtype, h.is_cuda) else 0            # tokens served by the packed kernel
    q, kv = M.qk_prep(ops.linear(h, w["wqk"]), nh, d, w["q_norm"], w["k_norm"], w["freq"], kp, vp, b, cfg.rms_norm_eps, tl > 0 and b.gather is None)
    out = []
    if tl:
        if b.gather is None:
            k, v, cu_k = kv[0][:tl], kv[1][:tl], b.cu[:b.n_long + 1]
        else:
            rows, cu_k = b.gather[view]
            k, v = M.gather_keys(kp, vp, rows)
        out.append(M.window_attention_varlen(q[:tl], k, v, b.cu[:b.n_long + 1], cu_k, scale, *view))
    if tl < t:
        lo = b.n_long if tl else 0
        seq_of = None if b.seq_of is None or tl else b.seq_of[tl:]
        out.append(M.window_attention(q[tl:], kp, vp, b.table[lo:], seq_of, b.kv_len[tl:], scale, *view, b.max_len))
    o = out[0] if len(out) == 1 else torch.cat(out)
    return o[..., :d].reshape(t, nh * d)


def _diff(cfg: ModelConfig, m: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch) -> torch.Tensor:
    nh, t, window = m["heads"], b.tokens, m["window"]
    kp, vp, eps = cache["k_pool"], cache["v_pool"], cfg.rms_norm_eps
    mix = M.MapMix(w["lam"], float(m["diff"]), eps, m["vdim"], m["dim"])
    tl = b.t_long if packs(m, h.dtype, h.is_cuda) else 0            # tokens served by the packed kernel
    q, kv = M.map_prep(ops.linear(h, w["wqkv"]), w["b_qkv"], nh, m["dim"], m["vdim"], w["q_norm"], w["k_norm"], w["freq"], kp, vp, b, eps,
                       tl > 0 and b.gather is None)
    out = []
    if tl:
        if b.gather is None:
            k, v, cu_k = kv[0][:tl], kv[1][:tl], b.cu[:b.n_long + 1]
        else:
            rows, cu_k = b.gather[window, 0]
            k, v = M.gather_keys(kp, vp, rows)
        out.append(M.map_attention_varlen(q[:tl], k, v, b.cu[:b.n_long + 1], cu_k, float(m["scale"]), window, mix))
    if tl < t:
        lo = b.n_long if tl else 0
        seq_of = None if b.seq_of is None or tl else b.seq_of[tl:]
        out.append(M.map_attention(q[tl:], kp, vp, b.table[lo:], seq_of, b.kv_len[tl:], float(m["scale"]), window, mix, b.max_len))
    return out[0] if len(out) == 1 else torch.cat(out)


_MIXERS = {"ssd": _ssd, "mlstm": _mlstm, "delta": _delta, "latent": _latent, "window": _window, "diff": _diff}


def _mixer(cfg: ModelConfig, lay: dict, w: dict, h: torch.Tensor, cache: dict, b: M.SpanBatch, bias: bool = True) -> torch.Tensor:
    """The mixer with its output product; ``bias=False``: an output bias (``b_o``) is left to the caller."""
    kind = lay["kind"]
    o = KINDS[kind].run(lay["sizes"], cfg.rms_norm_eps, w, h, cache, b) if kind in KINDS else _MIXERS[kind](cfg, lay["sizes"], w, h, cache, b)
    y = ops.linear(o, w["wo"])
    return y + w["b_o"].to(y.dtype) if bias and "b_o" in w else y


def layer_step(cfg: ModelConfig, i: int, w: dict, x: torch.Tensor, h: torch.Tensor, cache: dict, b: M.SpanBatch,
               w_next: torch.Tensor | None = None) -> torch.Tensor:
    """Layer ``i`` on one packed step.  x: fp32 residual stream, updated in place; h: what its mixer reads, in the activation dtype (x
    itself, or its norm ``pre1``).  Returns x in that dtype — or the norm of x with the weight ``w_next``, which is the next layer's
    ``pre1`` or the model's final norm."""
    lay, eps = cfg.layers[i], cfg.rms_norm_eps
    y = _mixer(cfg, lay, w, h, cache, b)
    if not lay["ff"]:
        return M.norm_add_(y, x, w["norm1"], eps, w_next)
    h = M.norm_add_(y, x, w["norm1"], eps, w.get("pre2"))
    a = M.linear_clamped_glu(h, w["wgu"], lay["limit"], lay["alpha"]) if lay.get("act") == "clamped_glu" else M.linear_gelu(h, w["wup"])
    return M.norm_add_(ops.linear(a, w["wdown"]), x, w["norm2"], eps, w_next)


def _feed_forward(cfg: ModelConfig, lay: dict, w: dict, h: torch.Tensor, beside: M.SpanBatch | None = None) -> tuple[torch.Tensor | None, M.Routed | None]:
    """(rows, routed rows that are still to be gathered) of a feed-forward.  With ``beside`` the shared expert of a step of single tokens runs next to
    the routed ones."""
    act = lay.get("act", "gelu")
    if act == "moe":
        glu = (float(lay["limit"]), float(lay["alpha"])) if "limit" in lay else None
        y = None
        with M.beside(h, beside) as side:
            if "swgu" in w:
                with side():
                    a = M.linear_silu_glu(h, w["swgu"]) if glu is None else M.linear_clamped_glu(h, w["swgu"], float(lay["shared_limit"]), glu[1])
                    y = ops.linear(a, w["swd"])
            routed = M.experts(h, w["router"], w["ewgu"], w["ewd"], lay["top"], glu, lay.get("router", ROUTERS[0]) == "softmax")
        return y, routed
    if act == "poly":
        a = M.poly_norm(ops.linear(h, w["wup"]), w["act"], cfg.rms_norm_eps)
    else:
        a = M.linear_clamped_glu(h, w["wgu"], lay["limit"], lay["alpha"]) if act == "clamped_glu" else M.linear_gelu(h, w["wup"])
    return ops.linear(a, w["wdown"]), None


def _conv_of(cfg: ModelConfig, w: dict, cache: dict) -> M.InputConv | None:
    return M.InputConv(w["conv1"], w.get("conv2"), cache["input"]) if cfg.input_conv else None


def _sublayers(cfg: ModelConfig, i: int, w: dict, h: tuple, cache: dict, b: M.SpanBatch) -> tuple:
    """(mixer rows, feed-forward rows, routed rows).  In single-token steps the two sublayers run on streams of their own: each is a chain of
    kernels that leave most of the GPU idle."""
    lay = cfg.layers[i]

    def mixer():
        return _mixer(cfg, lay, w, h[0], cache, b)

    if not lay["ff"]:
        return mixer(), None, None
    with M.beside(h[0], b) as side:
        with side():
            y2, routed = _feed_forward(cfg, lay, w, h[1])
        y1 = mixer()
    return y1, y2, routed


def _forward_parallel(cfg: ModelConfig, embed_w: dict, layer_w: list[dict], ids: torch.Tensor, caches: list[dict], b: M.SpanBatch,
                      final_norm: torch.Tensor | None) -> tuple[torch.Tensor, torch.Tensor]:
    n = len(layer_w)
    past, h = M.block_embed(ids, embed_w["embed"], n + 1 if cfg.depth_average else 1, layer_w[0]["pre1"], cfg.rms_norm_eps, cfg.layer_norm,
                            _conv_of(cfg, layer_w[0], caches[0]), b)
    x = None
    for i, w in enumerate(layer_w):
        last = i + 1 == n
        y1, y2, routed = _sublayers(cfg, i, w, h, caches[i], b)
        x, h = M.block_add(past, i, y1, y2, routed, w.get("ls1"), w.get("ls2"), layer_w[i - 1].get("depth") if i else None, w.get("depth"),
                           final_norm if last else layer_w[i + 1]["pre1"], cfg.rms_norm_eps, cfg.layer_norm,
                           None if last else _conv_of(cfg, layer_w[i + 1], caches[i + 1]), b, want_x=last)
    return x, h[0]


def _forward_streams(cfg: ModelConfig, embed_w: dict, layer_w: list[dict], ids: torch.Tensor, caches: list[dict], b: M.SpanBatch,
                     final_norm: torch.Tensor | None) -> tuple[torch.Tensor, torch.Tensor]:
    eps = cfg.rms_norm_eps
    subs = [(i, q) for i, lay in enumerate(cfg.layers) for q in ("1", "2") if q == "1" or lay["ff"]]
    x, h = M.streams_embed(ids, embed_w["embed"], cfg.embed_scale, cfg.streams, layer_w[0]["hc1.in"], layer_w[0]["pre1"], eps)
    for n, (i, q) in enumerate(subs):
        lay, w = cfg.layers[i], layer_w[i]
        y, routed = (_mixer(cfg, lay, w, h, caches[i], b, bias=False), None) if q == "1" else _feed_forward(cfg, lay, w, h, b)
        bias = w.get("b_o") if q == "1" else None
        hc = (w[f"hc{q}.mix"], w[f"hc{q}.out"])
        if n + 1 == len(subs):
            return M.streams_sum(x, y, bias, routed, *hc, final_norm, eps)
        j, r = subs[n + 1]
        x, h = M.streams_add(x, y, bias, routed, *hc, layer_w[j][f"hc{r}.in"], layer_w[j]["pre" + r], eps)


def forward(cfg: ModelConfig, embed_w: dict, layer_w: list[dict], ids: torch.Tensor, caches: list[dict], b: M.SpanBatch,
            final_norm: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """The stack on one packed step: (fp32 residual stream after the last layer, the same in the activation dtype — normed with
    ``final_norm`` when that is given)."""
    if cfg.parallel_block:
        return _forward_parallel(cfg, embed_w, layer_w, ids, caches, b, final_norm)
    if cfg.streams:
        return _forward_streams(cfg, embed_w, layer_w, ids, caches, b, final_norm)
    x, h = M.embed(ids, embed_w["embed"], layer_w[0].get("pre1"), cfg.rms_norm_eps)
    for i, w in enumerate(layer_w):
        h = layer_step(cfg, i, w, x, h, caches[i], b, layer_w[i + 1].get("pre1") if i + 1 < len(layer_w) else final_norm)
    return x, h
