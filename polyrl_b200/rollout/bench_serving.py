"""Serving throughput of mixer stacks beside the closest llama-family models of equal size: ``python bench.py --workload serving``.

Random weights.  Prefill: packed prompts through ``RolloutEngine.extend`` (device time of the step); decode: the engine's CUDA-graph
decode step; both timed with CUDA events after warm-up, weights (gigabytes) far larger than L2.  ``--kernels`` times the single kernels at
the same layer sizes, with L2 flushed between iterations, against their roofline: the larger of bytes / measured copy bandwidth and
FLOPs / measured bf16 GEMM rate.  ``--serving-design`` picks the mixer stack.
"""
from __future__ import annotations

import json
import os
from pathlib import Path

import torch


def _peaks() -> tuple[float, float, str]:
    p = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if p.exists():
        d = json.loads(p.read_text())
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def models(layers: int, design: str) -> dict:
    """The mixer stack and its closest stacks at the same width, feed-forward width and depth: llama with latent attention (MLA) beside
    ludesun, ludesun beside lanilix, llama beside all; beside mabedra lanilix and a llama stack with the same experts in the same layers; beside dubazen mabedra and the latter with experts in every layer."""
    from ..models import ModelConfig, get_model_config

    def stack(name):
        c = get_model_config(name)
        return ModelConfig(**{**c.to_dict(), "num_layers": layers, "layers": tuple(dict(c.layers[i % 4], weights_of=i) for i in range(layers))})

    hy = stack("ludesun-4b")
    base = dict(family="llama", vocab_size=hy.vocab_size, hidden_size=hy.hidden_size, intermediate_size=hy.intermediate_size, num_layers=layers, num_heads=32,
                max_position_embeddings=16384, rope_theta=500000.0, rms_norm_eps=1e-5, eos_token_id=-1)
    if design in ("mabedra", "dubazen"):
        moe = dict(num_experts=16, num_experts_per_tok=2, moe_intermediate_size=2048, shared_expert_intermediate_size=4096, norm_topk_prob=design == "dubazen",
                   dense_layers=tuple(range(0, layers, 4)) if design == "mabedra" else ())
    if design == "dubazen":
        return {"dubazen": stack("dubazen-7b"), "mabedra": stack("mabedra-7b"), "llama with experts": ModelConfig(**base, num_kv_heads=8, **moe)}
    if design == "mabedra":
        return {"mabedra": stack("mabedra-7b"), "lanilix": stack("lanilix-4b"), "llama": ModelConfig(**base, num_kv_heads=8),
                "llama with experts": ModelConfig(**base, num_kv_heads=8, **moe)}
    if design == "lanilix":
        return {"lanilix": stack("lanilix-4b"), "ludesun": hy, "llama": ModelConfig(**base, num_kv_heads=8)}
    return {"ludesun": hy,
            "llama": ModelConfig(**base, num_kv_heads=8),
            "mla": ModelConfig(**base, num_kv_heads=32, attn_type="mla", q_lora_rank=1536, kv_lora_rank=512, qk_nope_head_dim=128, qk_rope_head_dim=64,
                               v_head_dim=128)}


def _events(fn, iters: int, warmup: int, flush: torch.Tensor | None = None) -> float:
    """Median device milliseconds of ``fn``."""
    for _ in range(warmup):
        fn()
    ts = []
    for _ in range(iters):
        if flush is not None:
            flush.zero_()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        torch.cuda.synchronize()
        a.record()
        fn()
        b.record()
        torch.cuda.synchronize()
        ts.append(a.elapsed_time(b))
    return sorted(ts)[len(ts) // 2]


def run_models(args) -> list[dict]:
    from ..models import TransformerWeights
    from .engine import RolloutEngine

    dev, rows = torch.device("cuda"), []
    prefills = [(16, 1024), (2, 8192)]
    decodes = [(64, 1024), (128, 2048)]
    os.environ.setdefault("POLYRL_MOE_STATIC_DECODE", "1")        # llama-family experts: the decode form that can be captured
    for name, cfg in models(args.serving_layers, args.serving_design).items():
        w = TransformerWeights(cfg, device=dev, dtype=torch.bfloat16, init=True)
        n_params = cfg.num_params()
        for nseq, length in prefills:
            eng = RolloutEngine(cfg, dev, max_num_seqs=nseq, max_model_len=length + 64, kv_cache_tokens=nseq * (length + 64))
            eng.set_weights(w.embed, w.layers, w.head)
            g = torch.Generator().manual_seed(0)
            toks = [torch.randint(3, cfg.vocab_size, (length,), generator=g).tolist() for _ in range(nseq)]

            def step():
                rs = [eng.open() for _ in toks]
                eng.extend([(r, t, [length - 1]) for r, t in zip(rs, toks)])
                for r in rs:
                    eng.close(r)

            ms = _events(step, args.steps_serving, 3)
            rows.append({"model": name, "params": n_params, "phase": "prefill", "seqs": nseq, "len": length, "ms": round(ms, 3),
                         "tokens_per_s": round(nseq * length / ms * 1e3)})
            print(json.dumps(rows[-1]), flush=True)
            del eng
            torch.cuda.empty_cache()
        for nseq, ctx in decodes:
            eng = RolloutEngine(cfg, dev, max_num_seqs=nseq, max_model_len=ctx + 128, kv_cache_tokens=nseq * (ctx + 128) + 16)
            eng.set_weights(w.embed, w.layers, w.head)
            rs = [eng.open() for _ in range(nseq)]
            g = torch.Generator().manual_seed(1)
            for lo in range(0, nseq, 8):                      # prompts in, eight at a time
                eng.extend([(r, torch.randint(3, cfg.vocab_size, (ctx,), generator=g).tolist(), []) for r in rs[lo:lo + 8]])
            eng.extend([(r, [5], []) for r in rs])            # first decode step: captures the graph
            eng.st_active.fill_(1)
            ms = _events(lambda: eng._run_decode(nseq, sample=False), args.steps_serving, 3)
            rows.append({"model": name, "params": n_params, "phase": "decode", "seqs": nseq, "len": ctx, "ms": round(ms, 3),
                         "tokens_per_s": round(nseq / ms * 1e3)})
            print(json.dumps(rows[-1]), flush=True)
            for r in rs:
                eng.close(r)
            del eng
            torch.cuda.empty_cache()
        del w
        torch.cuda.empty_cache()
    return rows


class _Kernels:
    """Times single kernels against their roofline and collects the rows."""

    def __init__(self, args):
        self.dev, self.args, self.rows = torch.device("cuda"), args, []
        self.hbm, self.flops, self.kind = _peaks()
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=self.dev)

    def rnd(self, *s, dtype=torch.bfloat16, scale=1.0):
        return (torch.randn(*s, device=self.dev) * scale).to(dtype)

    def rec(self, name, like, shape, fn, nbytes, fl=0.0):
        fn()                                                  # (sets kernel attributes, sizes workspaces)
        for _ in range(6000):                                 # a third of a second of plain writes: the clocks recover from a GEMM under the power cap
            self.flush.zero_()
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()                        # launch latency of the Python wrappers stays out of the device time
        with torch.cuda.graph(graph):
            fn()
        ms = _events(graph.replay, self.args.steps_serving, 3, self.flush)
        del graph
        roof = max(nbytes / self.hbm, fl / self.flops) * 1e3
        self.rows.append({"kernel": name, "like": like, "shape": shape, "us": round(ms * 1e3, 1), "roofline_us": round(roof * 1e3, 1),
                          "of_" + self.kind: round(roof / ms, 3)})
        print(json.dumps(self.rows[-1]), flush=True)

    def batch(self, lens, start):
        """(SpanBatch of equal spans behind ``start`` earlier tokens, pages of the pool)."""
        from ..ops import mixers as M

        dev = self.dev
        n, t = len(lens), sum(lens)
        cu = torch.tensor([0] + lens, dtype=torch.int32).cumsum(0).to(torch.int32)
        seq_of = torch.repeat_interleave(torch.arange(n, dtype=torch.int32), torch.tensor(lens)).to(dev)
        long = lens[0] > 1
        pos = torch.cat([torch.arange(start, start + x) for x in lens]).to(dev)
        width = (start + max(lens) + 15) // 16
        table = (torch.arange(n * width).reshape(n, width) + 1).int().to(dev)
        kv = (table.long()[seq_of.long(), pos // 16] * 16 + pos % 16)
        return M.SpanBatch(cu=cu.to(dev), start=torch.full((n,), start, dtype=torch.int32, device=dev), slot=torch.arange(1, n + 1, device=dev), pos=pos,
                           kv_slot=kv, kv_len=(pos + 1).int(), table=table, seq_of=seq_of if long else None, n_long=n if long else 0,
                           t_long=t if long else 0, max_long=max(lens) if long else 0, max_len=start + max(lens)), width * n + 1


_SHAPES = (("16 x 1024", [1024] * 16, 0), ("2 x 8192", [8192] * 2, 0), ("decode 128 @ 2048", [1] * 128, 2047))


def run_kernels_lanilix(args) -> list[dict]:
    """Layer sizes of ``lanilix-4b``; ``like`` names the kernel of the same kind, ``existing:`` rows are those kernels."""
    from .. import ops
    from ..ops import mixers as M
    from ..ops.attention import attention_varlen

    C, K = ops.ext(), _Kernels(args)
    dev, rnd, rec = K.dev, K.rnd, K.rec
    W, FF = 4096, 14336
    f32 = dict(device=dev, dtype=torch.float32)
    for tag, lens, start in _SHAPES:
        b, blocks = K.batch(lens, start)
        t, n, L, dec = sum(lens), len(lens), lens[0], lens[0] == 1
        # ---- recurrences
        H, G, N, V = 32, 16, 128, 128
        ch = 2 * G * N + H * V
        cache = {"S": torch.zeros(n + 1, H, N, V, **f32)}
        c = rnd(t, ch)
        gates = M.Gates(rnd(t, H, dtype=torch.float32), rnd(t, H, dtype=torch.float32), torch.full((H,), -2.0, **f32), None, torch.linspace(-4, 1, H, **f32))
        # per token and head: three products with the state, and half a chunk of 64 earlier tokens for each of K K', Q K', the solve and P U
        rec("recurrence delta", "recurrence ssd", tag, lambda: M.scan(M.DELTA, c[:, :G * N], c[:, G * N:2 * G * N], c[:, 2 * G * N:], gates, N ** -0.5, cache, b),
            t * (2 * G * N * 2 + 2 * H * V * 2 + 2 * H * 4) + (2 if dec else 1) * n * H * N * V * 4, 0 if dec else t * H * (6 * N * V + 64 * (2 * N + 2 * V)))
        H2, V2, N2, G2 = 128, 64, 128, 8
        cache2 = {"S": torch.zeros(n + 1, H2, N2, V2, **f32)}
        q2, k2, v2 = rnd(t, G2 * N2), rnd(t, G2 * N2, scale=N2 ** -0.5), rnd(t, H2 * V2)
        gates2 = M.Gates(rnd(t, H2, dtype=torch.float32), None, torch.full((H2,), -2.0, **f32), None, torch.linspace(-2, 1, H2, **f32), torch.ones(H2, **f32))
        rec("existing: recurrence ssd", "recurrence ssd", tag, lambda: M.scan(M.SSD, q2, k2, v2, gates2, 1.0, cache2, b),
            t * (2 * G2 * N2 * 2 + 2 * H2 * V2 * 2 + H2 * 4) + (2 if dec else 1) * n * H2 * N2 * V2 * 4, 0 if dec else t * H2 * (64 * (N2 + V2) + 4 * N2 * V2))
        del cache2, q2, k2, v2, c
        p = rnd(t, ch + H * V)
        cw, cb, cst = torch.randn(4, ch, device=dev), torch.randn(ch, device=dev), torch.zeros(n + 1, 3, ch, device=dev, dtype=torch.bfloat16)
        rec("conv + silu, no bias", "conv + silu", tag, lambda: M.conv_silu(p[:, :ch], cw, None, cst, b), t * ch * 4 + n * 6 * ch * 2)
        rec("existing: conv + silu", "conv + silu", tag, lambda: M.conv_silu(p[:, :ch], cw, cb, cst, b), t * ch * 4 + n * 6 * ch * 2)
        y, gn = rnd(t, H * V), torch.ones(H * V, device=dev)
        rec("gated norm (silu last)", "gated norm", tag, lambda: M.gated_norm(y, p[:, ch:], gn, H, 1e-6, M.SILU_LAST), t * H * V * 6)
        rec("existing: gated norm (gate first)", "gated norm", tag, lambda: M.gated_norm(y, p[:, ch:], gn, 8, 1e-6, M.SILU_FIRST), t * H * V * 6)
        del cache, p, y
        # ---- attention
        H, G, D, rd = 32, 8, 128, 64
        qk = rnd(t, (H + G) * D)
        kp, vp = rnd(blocks, G, 16, D), rnd(blocks, G, 16, D)
        wq, wk, freq = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev), M.rope_frequencies(rd, 5e5, dev)
        rec("query / key norm, rotation, cache write", "latent rows", tag, lambda: M.qk_prep(qk, H, D, wq, wk, freq, kp, vp, b, 1e-6, not dec),
            t * ((H + G) * D * 2 + (H + (2 if dec else 4) * G) * D * 2))
        r, lr, qr = 512, 64, 1536
        pool, a = rnd(blocks, 1, 16, r + lr), rnd(t, qr + r + lr)
        w1, w2, fr = torch.ones(qr, device=dev), torch.ones(r, device=dev), M.rope_frequencies(lr, 1e4, dev)
        rec("existing: latent rows", "latent rows", tag, lambda: M.latent_prep(a, w1, w2, fr, pool, b, 1e-5, not dec), t * ((qr + r + lr) * 4 + (0 if dec else (r + lr) * 2)))
        del pool, a, qk
        q = rnd(t, H, D)
        k, v = (None, None) if dec else (rnd(t, G, D), rnd(t, G, D))
        for window, keep in ((4096, 4), (512, 4)):
            if dec:
                seen = min(2048, window + keep)
                rec(f"paged windowed attention, window {window}", "paged decode", tag,
                    lambda: M.window_attention(q, kp, vp, b.table, None, b.kv_len, 0.088, window, keep, b.max_len), t * seen * G * D * 4)
            else:
                pairs = sum(min(i + 1, window + min(keep, max(0, i + 1 - window))) for i in range(L))
                rec(f"packed windowed attention, window {window}", "packed attention", tag,
                    lambda: M.window_attention_varlen(q, k, v, b.cu, b.cu, 0.088, window, keep), t * (2 * H + 2 * G) * D * 2, n * pairs * H * 4 * D)
        if dec:
            rec("existing: paged decode (GQA 32/8)", "paged decode", tag,
                lambda: ops.paged_decode_attention(q.view(t, H * D), kp, vp, b.table, b.kv_len, H, G, D, 0.088, max_len=2048), t * 2048 * G * D * 4)
        else:
            rec("existing: attention_varlen (GQA 32/8)", "packed attention", tag, lambda: attention_varlen(q, k, v, b.cu, L, True, 0.088),
                t * (2 * H + 2 * G) * D * 2, n * L * L / 2 * H * 4 * D)
        del kp, vp, q, k, v
        # ---- rows and feed-forward
        x32, yb, wn, hb = torch.randn(t, W, device=dev), rnd(t, W), torch.ones(W, device=dev), rnd(t, W)
        rec("norm + residual add + next norm", "norm + residual add", tag, lambda: M.norm_add_(yb, x32, wn, 1e-6, wn), t * W * 12)
        rec("existing: norm + residual add", "norm + residual add", tag, lambda: M.norm_add_(yb, x32, wn, 1e-6), t * W * 12)
        wb = torch.ones(W, device=dev, dtype=torch.bfloat16)
        rec("existing: add_rmsnorm", "norm + residual add", tag, lambda: C.add_rmsnorm_(hb, yb, wb, 1e-5), t * W * 8)
        gu = rnd(2 * FF, W, scale=W ** -0.5)
        rec("gate / up + clamped glu", "gate / up + swiglu", tag, lambda: M.linear_clamped_glu(hb, gu, 7.0, 1.702), (t * W + 2 * FF * W + t * FF) * 2, 4.0 * t * W * FF)
        rec("existing: gate / up + swiglu", "gate / up + swiglu", tag, lambda: ops.linear_swiglu(hb, gu), (t * W + 2 * FF * W + t * FF) * 2, 4.0 * t * W * FF)
        emb, ids = rnd(128256, W), torch.randint(0, 128256, (t,), device=dev)
        rec("embedding + norm", "norm + residual add", tag, lambda: M.embed(ids, emb, wn, 1e-6), t * W * 8)
        del x32, yb, hb, gu, emb
        torch.cuda.empty_cache()
    return K.rows


def run_kernels_mabedra(args) -> list[dict]:
    """Layer sizes of ``mabedra-7b``."""
    from .. import ops
    from ..ops import mixers as M
    from ..ops.attention import attention_varlen

    C, K = ops.ext(), _Kernels(args)
    dev, rnd, rec = K.dev, K.rnd, K.rec
    W, FF = 4096, 14336
    f32 = dict(device=dev, dtype=torch.float32)
    for tag, lens, start in _SHAPES:
        b, blocks = K.batch(lens, start)
        t, n, L, dec = sum(lens), len(lens), lens[0], lens[0] == 1
        # ---- attention
        H, G, D, V, rd = 32, 8, 64, 128, 64
        kp, vp = rnd(blocks, G, 16, 2 * D), rnd(blocks, G, 16, V)
        cols = 2 * (H + G) * D + G * V
        p, bias, wn, freq = rnd(t, cols), torch.zeros(cols, **f32), torch.ones(D, **f32), M.rope_frequencies(rd, 5e5, dev)
        rec("map rows: bias, norms, rotation, cache write", "query / key rows", tag, lambda: M.map_prep(p, bias, H, D, V, wn, wn, freq, kp, vp, b, 1e-6, not dec),
            t * (cols * 2 + 2 * H * D * 2 + (1 if dec else 2) * G * (2 * D + V) * 2))
        qk, wq, wk = rnd(t, (H + G) * 128), torch.ones(H * 128, **f32), torch.ones(G * 128, **f32)
        rec("existing: query / key norm, rotation, cache write", "query / key rows", tag, lambda: M.qk_prep(qk, H, 128, wq, wk, freq, kp, vp, b, 1e-6, not dec),
            t * ((H + G) * 128 * 2 + (H + (2 if dec else 4) * G) * 128 * 2))
        del p, qk
        mix = M.MapMix(torch.full((1,), 0.5, **f32), 0.5, 1e-6, V, D)
        q2, q1 = rnd(t, 2 * H, D), rnd(t, H, 128)
        k2, v, k1 = (None,) * 3 if dec else (rnd(t, G, 2 * D), rnd(t, G, V), rnd(t, G, 128))
        for window in (4096, 512):
            if dec:
                rec(f"paged differential attention, window {window}", "paged decode", tag,
                    lambda: M.map_attention(q2, kp, vp, b.table, None, b.kv_len, 0.125, window, mix, b.max_len), t * min(2048, window) * G * (2 * D + V) * 2)
                rec(f"existing: paged windowed attention, window {window}", "paged decode", tag,
                    lambda: M.window_attention(q1, kp, vp, b.table, None, b.kv_len, 0.088, window, 0, b.max_len), t * min(2048, window) * G * 256 * 2)
            else:
                pairs = sum(min(i + 1, window) for i in range(L))
                rec(f"packed differential attention, window {window}", "packed attention", tag,
                    lambda: M.map_attention_varlen(q2, k2, v, b.cu, b.cu, 0.125, window, mix), t * (2 * H * D + H * V + G * (2 * D + V)) * 2,
                    n * pairs * H * 2 * (2 * D + 2 * V))
                rec(f"existing: packed windowed attention, window {window}", "packed attention", tag,
                    lambda: M.window_attention_varlen(q1, k1, v, b.cu, b.cu, 0.088, window, 0), t * (2 * H + 2 * G) * 128 * 2, n * pairs * H * 4 * 128)
        if not dec:
            rec("existing: attention_varlen (GQA 32/8)", "packed attention", tag, lambda: attention_varlen(q1, k1, v, b.cu, L, True, 0.088),
                t * (2 * H + 2 * G) * 128 * 2, n * L * L / 2 * H * 4 * 128)
        del kp, vp, q1, q2, k1, k2, v
        # ---- rows
        emb, ids, wn = rnd(128256, W), torch.randint(0, 128256, (t,), device=dev), torch.ones(W, **f32)
        cw, cst = torch.randn(4, W, **f32), torch.zeros(n + 1, 3, W, device=dev, dtype=torch.bfloat16)
        conv = M.InputConv(cw, cw.clone(), cst)
        fused = conv if dec else None                           # single-token steps: the block kernels end in the convolutions
        extra = n * W * (2 + 12) if dec else 0
        rec("embedding + norm" + (" + convolutions" if dec else ""), "norm + residual add", tag, lambda: M.block_embed(ids, emb, 1, wn, 1e-6, True, fused, b), t * W * 8 + extra)
        rec("existing: embedding + norm", "norm + residual add", tag, lambda: M.embed(ids, emb, wn, 1e-6), t * W * 8)
        del emb
        y1, y2, h = rnd(t, W), rnd(t, W), rnd(t, W)
        if not dec:
            rec("two input convolutions", "conv + silu", tag, lambda: M.input_conv(h, conv, b), t * W * 6 + n * 6 * W * 2)
            rec("existing: conv + silu", "conv + silu", tag, lambda: M.conv_silu(h, cw, None, cst, b), t * W * 4 + n * 6 * W * 2)
        past = torch.randn(17, t, W, **f32)
        for i in (0, 5, 15):
            a = torch.full((i + 2,), 0.1, **f32)
            rec(f"block results, average over {i + 2}, next norm" + (" + convolutions" if dec else ""), "norm + residual add", tag,
                lambda: M.block_add(past, i, y1, y2, None, wn, wn, a[1:] if i else None, a, wn, 1e-6, True, fused, b), t * W * (4 * (i + 2) + 6) + extra)
        del past
        x32 = torch.randn(t, W, **f32)
        rec("existing: norm + residual add + next norm", "norm + residual add", tag, lambda: M.norm_add_(y1, x32, wn, 1e-6, wn), t * W * 12)
        z, act = rnd(t, FF), torch.tensor([0.3, 0.3, 0.3, 0.1], **f32)
        rec("polynomial activation", "gated norm", tag, lambda: M.poly_norm(z, act, 1e-6), t * FF * 4)
        z2, gn = rnd(t, FF), torch.ones(FF, **f32)
        rec("existing: gated norm (gate first)", "gated norm", tag, lambda: M.gated_norm(z, z2, gn, 1, 1e-6, M.SILU_FIRST), t * FF * 6)
        del z, z2, x32, y2
        # ---- experts
        E, top, F = 16, 2, 2048
        router = rnd(E, W, scale=W ** -0.5)
        wgu, wd = rnd(E * 2 * F, W, scale=W ** -0.5), rnd(E * W, F, scale=F ** -0.5)
        logits = M.linear_f32(h, router)
        ctr = M._counter(dev, E + 1, "route")
        pick, score, rank, plan = C.mix_route(logits, top, ctr)
        xr, pos = C.mix_expert_rows(h, pick, score, rank, plan, E)
        a = C.gemm_experts(xr, wgu, plan, E, True)
        rec("routing", "norm + residual add", tag, lambda: C.mix_route(logits, top, ctr), t * (E * 4 + top * 12))
        rec("rows in the experts' order", "norm + residual add", tag, lambda: C.mix_expert_rows(h, pick, score, rank, plan, E), t * W * 2 * (1 + top))
        rec("experts: gate / up + silu glu", "gate / up + swiglu", tag, lambda: C.gemm_experts(xr, wgu, plan, E, True),
            (E * 2 * F * W + t * top * (W + F)) * 2, 4.0 * t * top * W * F)
        rec("experts: down", "down projection", tag, lambda: C.gemm_experts(a, wd, plan, E, False), (E * F * W + t * top * (W + F)) * 2, 2.0 * t * top * W * F)
        routed = M.Routed(C.gemm_experts(a, wd, plan, E, False), pos)
        past, a2 = torch.randn(7, t, W, **f32), torch.full((7,), 0.1, **f32)
        ys = rnd(t, W)
        rec("block results with routed rows, average over 7" + (" + convolutions" if dec else ""), "norm + residual add", tag,
            lambda: M.block_add(past, 5, y1, ys, routed, wn, wn, a2[1:], a2, wn, 1e-6, True, fused, b), t * W * (28 + 6 + 2 * top) + extra)
        del past, xr, a, routed
        gu, dn, g = rnd(2 * top * F, W, scale=W ** -0.5), rnd(W, top * F, scale=W ** -0.5), rnd(t, top * F)
        rec("existing: gate / up + swiglu, dense of the active width", "gate / up + swiglu", tag, lambda: ops.linear_swiglu(h, gu),
            (t * W + 2 * top * F * W + t * top * F) * 2, 4.0 * t * top * W * F)
        rec("existing: down projection, dense of the active width", "down projection", tag, lambda: ops.linear(g, dn), (t * W + top * F * W + t * top * F) * 2,
            2.0 * t * top * W * F)
        del gu, dn, g, wgu, wd, y1, h
        torch.cuda.empty_cache()
    return K.rows


def run_kernels_dubazen(args) -> list[dict]:
    """Layer sizes of ``dubazen-7b``."""
    from .. import ops
    from ..ops import mixers as M
    from ..ops.attention import attention_varlen

    C, K = ops.ext(), _Kernels(args)
    dev, rnd, rec = K.dev, K.rnd, K.rec
    W = 4096
    f32 = dict(device=dev, dtype=torch.float32)
    for tag, lens, start in _SHAPES:
        b, blocks = K.batch(lens, start)
        t, n, L, dec = sum(lens), len(lens), lens[0], lens[0] == 1
        rw = (2 if dec else 1) * n
        # ---- recurrences
        I, N = 8192, 16
        p, x, dt, bc = rnd(t, 2 * I), rnd(t, I), rnd(t, I, dtype=torch.float32), rnd(t, 256 + 2 * N)
        vec, a_neg, state = torch.full((I,), -2.0, **f32), -torch.arange(1, N + 1, **f32).expand(I, N).contiguous(), torch.zeros(n + 1, I, N, **f32)
        rec("selective scan", "recurrence ssd", tag, lambda: M.selective_scan(x, dt, bc[:, 256:256 + N], bc[:, 256 + N:], p[:, I:], vec, a_neg, vec, state, b),
            t * (I * 10 + 4 * N) + rw * I * N * 4)
        cw, cb, cst = torch.randn(4, I, device=dev), torch.randn(I, device=dev), torch.zeros(n + 1, 3, I, device=dev, dtype=torch.bfloat16)
        rec("existing: conv + silu", "conv + silu", tag, lambda: M.conv_silu(p[:, :I], cw, cb, cst, b), t * I * 4 + n * 6 * I * 2)
        del p, x, dt, bc, state
        H, N, V = 16, 128, 256
        cache, q, k, v, z = {"S": torch.zeros(n + 1, H, N, V, **f32)}, rnd(t, H * N), rnd(t, H * N), rnd(t, H * V), rnd(t, H * N, dtype=torch.float32)
        gates = M.Gates(z, b0=torch.full((H * N,), 3.0, **f32), cap=16.0)
        # per token and head: two products with the state, half a chunk of 64 earlier tokens for each of Q K' and P V
        rec("recurrence gla", "recurrence delta", tag, lambda: M.scan(M.GLA, q, k, v, gates, N ** -0.5, cache, b), t * H * (2 * N * 2 + 2 * V * 2 + N * 4) + rw * H * N * V * 4,
            0 if dec else t * H * (4 * N * V + 64 * (N + V)))
        o, g, gn = rnd(t, H * V), rnd(t, H * V), torch.ones(H * V, device=dev)
        rec("existing: gated norm per head", "gated norm", tag, lambda: M.gated_norm(o, g, gn, H, 1e-6, M.SILU_LAST), t * H * V * 6)
        del z
        H, N, V = 32, 128, 128
        q, k, v, cache = rnd(t, H * N), rnd(t, H * N), rnd(t, H * V), {"S": torch.zeros(n + 1, H, N, V, **f32)}
        light = M.Gates(a_log=torch.linspace(-1, -0.001, H, **f32), raw=dec)
        rec("recurrence with constant decay" + (" + silu" if dec else ""), "recurrence ssd", tag, lambda: M.scan(M.DECAY, q, k, v, light, 1.0, cache, b),
            t * H * (2 * N + 2 * V) * 2 + rw * H * N * V * 4, 0 if dec else t * H * (64 * (N + V) + 4 * N * V))
        gates = M.Gates(rnd(t, H, dtype=torch.float32), rnd(t, H, dtype=torch.float32), torch.full((H,), -2.0, **f32), None, torch.linspace(-4, 1, H, **f32))
        rec("existing: recurrence delta", "recurrence delta", tag, lambda: M.scan(M.DELTA, q, k, v, gates, N ** -0.5, cache, b),
            t * (2 * H * N * 2 + 2 * H * V * 2 + 2 * H * 4) + rw * H * N * V * 4, 0 if dec else t * H * (6 * N * V + 64 * (2 * N + 2 * V)))
        H2, V2, N2, G2 = 128, 64, 128, 8
        cache2 = {"S": torch.zeros(n + 1, H2, N2, V2, **f32)}
        q2, k2, v2 = rnd(t, G2 * N2), rnd(t, G2 * N2, scale=N2 ** -0.5), rnd(t, H2 * V2)
        gates2 = M.Gates(rnd(t, H2, dtype=torch.float32), None, torch.full((H2,), -2.0, **f32), None, torch.linspace(-2, 1, H2, **f32), torch.ones(H2, **f32))
        rec("existing: recurrence ssd", "recurrence ssd", tag, lambda: M.scan(M.SSD, q2, k2, v2, gates2, 1.0, cache2, b),
            t * (2 * G2 * N2 * 2 + 2 * H2 * V2 * 2 + H2 * 4) + rw * H2 * N2 * V2 * 4, 0 if dec else t * H2 * (64 * (N2 + V2) + 4 * N2 * V2))
        if not dec:
            hb, wq = rnd(t, W), rnd(H * (2 * N + V), W, scale=W ** -0.5)
            rec("projection + silu", "gate / up + swiglu", tag, lambda: M.linear_silu(hb, wq), (t * W + wq.numel() + t * wq.shape[0]) * 2, 2.0 * t * wq.numel())
            rec("existing: projection + gelu", "gate / up + swiglu", tag, lambda: M.linear_gelu(hb, wq), (t * W + wq.numel() + t * wq.shape[0]) * 2, 2.0 * t * wq.numel())
            del hb, wq
        del cache, cache2, q, k, v, q2, k2, v2, o
        # ---- attention
        H, G, D, rd = 32, 8, 128, 64
        cols = (H + 2 * G) * D
        p, bias, freq, vfreq = rnd(t, cols), torch.zeros(cols, **f32), M.rope_frequencies(rd, 5e5, dev), M.rope_frequencies(D, 5e5, dev)
        kp, vp, sink = rnd(blocks, G, 16, D), rnd(blocks, G, 16, D), torch.zeros(H, **f32)
        rec("attention rows: bias, rotation, norms, rotated values, cache write", "query / key rows", tag, lambda: M.turn_prep(p, bias, H, D, D, freq, vfreq, kp, vp, b, 1e-6, not dec),
            t * (cols * 2 + H * D * 2 + (1 if dec else 2) * G * 2 * D * 2))
        wq, wk = torch.ones(H * D, **f32), torch.ones(G * D, **f32)
        rec("existing: query / key norm, rotation, cache write", "query / key rows", tag, lambda: M.qk_prep(p, H, D, wq, wk, freq, kp, vp, b, 1e-6, not dec),
            t * ((H + G) * D * 2 + (H + (2 if dec else 4) * G) * D * 2))
        q, o, gate = rnd(t, H, D), rnd(t, H, D), rnd(t, H * D)
        out = torch.empty_like(gate)
        rec("outputs turned back + gate", "gated norm", tag, lambda: M.turn_back(o, gate, vfreq, b.pos, 1.0, out), t * H * D * 6)
        if dec:
            rec("paged attention + sink", "paged decode", tag, lambda: M.sink_attention(q, kp, vp, b.table, None, b.kv_len, 0.088, sink, 2048), t * 2048 * G * D * 4)
            rec("existing: paged decode (GQA 32/8)", "paged decode", tag,
                lambda: ops.paged_decode_attention(q.view(t, H * D), kp, vp, b.table, b.kv_len, H, G, D, 0.088, max_len=2048), t * 2048 * G * D * 4)
        else:
            k, v = rnd(t, G, D), rnd(t, G, D)
            rec("packed attention + sink", "packed attention", tag, lambda: M.sink_attention_varlen(q, k, v, b.cu, b.cu, 0.088, sink), t * (2 * H + 2 * G) * D * 2,
                n * L * L / 2 * H * 4 * D)
            rec("existing: attention_varlen (GQA 32/8)", "packed attention", tag, lambda: attention_varlen(q, k, v, b.cu, L, True, 0.088), t * (2 * H + 2 * G) * D * 2,
                n * L * L / 2 * H * 4 * D)
            del k, v
        del p, kp, vp, q, o, gate, out
        # ---- residual streams
        S = 4
        emb, ids, one, wn = rnd(128256, W), torch.randint(0, 128256, (t,), device=dev), torch.ones(1, **f32), torch.ones(W, **f32)
        win, mix, ov = torch.full((S,), 0.25, **f32), torch.eye(S, **f32), torch.ones(S, **f32)
        rec("embedding + norm, streams", "norm + residual add", tag, lambda: M.streams_embed(ids, emb, 64.0, S, win, one, 1e-6), t * W * 8)
        rec("existing: embedding + norm", "norm + residual add", tag, lambda: M.embed(ids, emb, wn, 1e-6), t * W * 8)
        del emb
        xs, y = torch.randn(t, S, W, **f32), rnd(t, W)
        rec("four streams: mix, add, next norm", "norm + residual add", tag, lambda: M.streams_add(xs, y, wn, None, mix, ov, win, one, 1e-6), t * W * (8 * S + 4))
        x1 = xs[:, :1].contiguous()
        rec("four streams, first sublayer", "norm + residual add", tag, lambda: M.streams_add(x1, y, wn, None, mix, ov, win, one, 1e-6), t * W * (4 + 4 * S + 4))
        rec("four streams, sum and norm", "norm + residual add", tag, lambda: M.streams_sum(xs, y, wn, None, mix, ov, wn, 1e-6), t * W * (4 * S + 8))
        x32 = torch.randn(t, W, **f32)
        rec("existing: norm + residual add + next norm", "norm + residual add", tag, lambda: M.norm_add_(y, x32, wn, 1e-6, wn), t * W * 12)
        del x32, x1
        # ---- experts
        E, top, F = 16, 2, 2048
        h, router = rnd(t, W), rnd(E, W, scale=W ** -0.5)
        wgu, wd = rnd(E * 2 * F, W, scale=W ** -0.5), rnd(E * W, F, scale=F ** -0.5)
        logits, ctr = M.linear_f32(h, router), M._counter(dev, E + 1, "route")
        pick, score, rank, plan = C.mix_route(logits, top, ctr, True)
        xr, pos = C.mix_expert_rows(h, pick, None, rank, plan, E)
        a = C.gemm_experts(xr, wgu, plan, E, 2, 7.0, 1.702)
        rec("routing, softmax", "routing", tag, lambda: C.mix_route(logits, top, ctr, True), t * (E * 4 + top * 12))
        rec("existing: routing, sigmoid", "routing", tag, lambda: C.mix_route(logits, top, ctr), t * (E * 4 + top * 12))
        rec("rows in the experts' order", "rows in the experts' order", tag, lambda: C.mix_expert_rows(h, pick, None, rank, plan, E), t * W * 2 * (1 + top))
        rec("experts: gate / up + clamped glu", "experts: gate / up", tag, lambda: C.gemm_experts(xr, wgu, plan, E, 2, 7.0, 1.702), (E * 2 * F * W + t * top * (W + F)) * 2,
            4.0 * t * top * W * F)
        rec("existing: experts: gate / up + silu glu", "experts: gate / up", tag, lambda: C.gemm_experts(xr, wgu, plan, E, 1), (E * 2 * F * W + t * top * (W + F)) * 2,
            4.0 * t * top * W * F)
        rec("existing: experts: down", "experts: down", tag, lambda: C.gemm_experts(a, wd, plan, E, 0), (E * F * W + t * top * (W + F)) * 2, 2.0 * t * top * W * F)
        routed = M.Routed(C.gemm_experts(a, wd, plan, E, 0), pos, score)
        rec("four streams with routed rows", "norm + residual add", tag, lambda: M.streams_add(xs, y, None, routed, mix, ov, win, one, 1e-6), t * W * (8 * S + 4 + 2 * top))
        del xs, y, xr, a, routed, wgu, wd, h
        torch.cuda.empty_cache()
    return K.rows


def run_kernels(args) -> list[dict]:
    from .. import ops
    from ..models import get_model_config, mla
    from ..ops import mixers as M

    C, K = ops.ext(), _Kernels(args)
    dev, rnd, rec, bf = K.dev, K.rnd, K.rec, torch.bfloat16
    W, FF = 4096, 14336
    for tag, lens, start in _SHAPES:
        b, blocks = K.batch(lens, start)
        t, n, dec = sum(lens), len(lens), lens[0] == 1
        st_rw = 2 if dec else 1
        # ---- recurrences
        H, V, N, G = 128, 64, 128, 8
        cache = {"S": torch.zeros(n + 1, H, N, V, device=dev)}
        q, k, v = rnd(t, G * N), rnd(t, G * N, scale=N ** -0.5), rnd(t, H * V)
        gates = M.Gates(rnd(t, H, dtype=torch.float32), None, torch.full((H,), -2.0, device=dev), None, torch.linspace(-2, 1, H, device=dev), torch.ones(H, device=dev))
        rec("recurrence ssd", "attention", tag, lambda: M.scan(M.SSD, q, k, v, gates, 1.0, cache, b),
            t * (2 * G * N * 2 + 2 * H * V * 2 + H * 4) + st_rw * n * H * N * V * 4, 0 if dec else t * H * (64 * (N + V) + 4 * N * V))
        cw, cb = torch.randn(4, H * V + 2 * G * N, device=dev), torch.randn(H * V + 2 * G * N, device=dev)
        cst, xc = torch.zeros(n + 1, 3, H * V + 2 * G * N, device=dev, dtype=bf), rnd(t, 2 * H * V + 2 * G * N)
        ch = H * V + 2 * G * N
        rec("conv + silu", "rope", tag, lambda: M.conv_silu(xc[:, H * V:], cw, cb, cst, b), t * ch * 4 + n * 6 * ch * 2)
        y, z, gn = rnd(t, H * V), xc[:, :H * V], torch.ones(H * V, device=dev)
        rec("gated norm (gate first)", "rmsnorm", tag, lambda: M.gated_norm(y, z, gn, 8, 1e-5, M.SILU_FIRST), t * H * V * 6)
        del cache, q, k, v, xc, y
        H, V, N = 8, 512, 256
        cache = {"S": torch.zeros(n + 1, H, N, V, device=dev), "n": torch.zeros(n + 1, H, N, device=dev), "m": torch.zeros(n + 1, H, device=dev)}
        p = rnd(t, 2 * H * N + 2 * H * V)
        g = rnd(t, 2 * H, dtype=torch.float32)
        gates = M.Gates(g[:, :H], g[:, H:], torch.zeros(H, device=dev), torch.full((H,), 3.0, device=dev), cap=15.0)
        rec("recurrence mlstm", "attention", tag, lambda: M.scan(M.MLSTM, p[:, :H * N], p[:, H * N:2 * H * N], p[:, 2 * H * N:2 * H * N + H * V], gates, N ** -0.5, cache, b),
            t * (2 * H * N * 2 + 2 * H * V * 2 + 2 * H * 4) + st_rw * n * H * N * V * 4, 0 if dec else t * H * (64 * (N + V) + 4 * N * V))
        y, gn = rnd(t, H * V), torch.ones(H * V, device=dev)
        rec("gated norm (gate last)", "rmsnorm", tag, lambda: M.gated_norm(y, p[:, 2 * H * N + H * V:], gn, 8, 1e-5, M.SIGMOID_LAST), t * H * V * 6)
        del cache, p, y
        # ---- latent attention
        H, d, rd, V, r, qr = 32, 128, 64, 128, 512, 1536
        pool = rnd(blocks, 1, 16, r + rd)
        freq = M.rope_frequencies(rd, 1e4, dev)
        a, q = rnd(t, qr + r + rd), rnd(t, H, d + rd)
        wq, wkv, sink = torch.ones(qr, device=dev), torch.ones(r, device=dev), torch.zeros(H, device=dev)
        rec("latent rows", "rmsnorm", tag, lambda: M.latent_prep(a, wq, wkv, freq, pool, b, 1e-5, not dec), t * ((qr + r + rd) * 4 + (0 if dec else (r + rd) * 2)))
        rec("rope of queries", "rope", tag, lambda: M.rope_(q, d, freq, b.pos), t * H * rd * 4)
        if dec:
            q_lat = rnd(H, t, r)
            rec("paged latent attention + sink", "paged attention", tag, lambda: M.latent_attention(q_lat, q, d, pool, b.table, None, b.kv_len, sink, 0.07, 2048),
                t * 2048 * (r + rd) * 2, t * 2048 * H * 2 * (2 * r + rd))
            qa = torch.cat([q_lat.transpose(0, 1), q[..., d:]], -1).contiguous()
            rec("existing: mla.paged_latent_attention", "paged attention", tag, lambda: mla.paged_latent_attention(qa, pool, b.table, b.kv_len, r, 0.07),
                t * 2048 * (r + rd) * 2, t * 2048 * H * 2 * (2 * r + rd))
            kc, vc = rnd(blocks, 8, 16, 128), rnd(blocks, 8, 16, 128)
            qq = rnd(t, 32 * 128)
            rec("existing: paged_decode (GQA 32/8)", "paged attention", tag,
                lambda: ops.paged_decode_attention(qq, kc, vc, b.table, b.kv_len, 32, 8, 128, 0.088, max_len=2048), t * 2048 * 8 * 128 * 4)
            del kc, vc
        else:
            from ..ops.attention import attention_varlen

            kk, vv = rnd(t, H, d + rd), rnd(t, H, V)
            L = lens[0]
            fl = n * L * L / 2 * H * 2 * (d + rd + V)
            rec("packed attention 192 / 128 + sink", "attention", tag, lambda: M.sink_attention_varlen(q, kk, vv, b.cu, b.cu, 0.07, sink),
                t * H * (2 * (d + rd) + 2 * V) * 2, fl)
            vp = torch.nn.functional.pad(vv, (0, rd))
            rec("existing: attention_varlen of the MLA stack", "attention", tag, lambda: attention_varlen(q, kk, vp, b.cu, L, True, 0.07),
                t * H * (2 * (d + rd) + 2 * V) * 2, fl)
            q8, k8, v8 = rnd(t, 32, 128), rnd(t, 8, 128), rnd(t, 8, 128)
            rec("existing: attention_varlen (GQA 32/8)", "attention", tag, lambda: attention_varlen(q8, k8, v8, b.cu, L, True, 0.088),
                t * 80 * 128 * 2, n * L * L / 2 * 32 * 2 * 256)
            del kk, vv, vp, q8, k8, v8
        del pool, a, q
        # ---- rows and feed-forward
        x32, yb, wn, hb = torch.randn(t, W, device=dev), rnd(t, W), torch.ones(W, device=dev), rnd(t, W)
        rec("norm + residual add", "rmsnorm", tag, lambda: M.norm_add_(yb, x32, wn, 1e-5), t * W * 12)
        wb = torch.ones(W, device=dev, dtype=bf)
        rec("existing: add_rmsnorm", "rmsnorm", tag, lambda: C.add_rmsnorm_(hb, yb, wb, 1e-5), t * W * 8)
        up, gu = rnd(FF, W, scale=W ** -0.5), rnd(2 * FF, W, scale=W ** -0.5)
        rec("up projection + gelu", "gate/up + swiglu", tag, lambda: M.linear_gelu(hb, up), (t * W + FF * W + t * FF) * 2, 2.0 * t * W * FF)
        rec("existing: gate/up + swiglu", "gate/up + swiglu", tag, lambda: ops.linear_swiglu(hb, gu), (t * W + 2 * FF * W + t * FF) * 2, 4.0 * t * W * FF)
        qkv = rnd(t, 48 * 128)
        ll = get_model_config("llama3-8b", max_position_embeddings=16384)
        from ..models.transformer import rope_tables

        cos, sin = rope_tables(ll, dev)
        rec("existing: rope (GQA 32/8)", "rope", tag, lambda: ops.apply_rope(qkv, b.pos, cos, sin, 32, 8, 128), t * 40 * 128 * 4)
        del x32, yb, hb, up, gu, qkv
        torch.cuda.empty_cache()
    return K.rows


@torch.no_grad()
def main(args) -> int:
    if not torch.cuda.is_available():
        print(json.dumps({"error": "the serving workload needs a CUDA device"}))
        return 1
    args.steps_serving = max(5, args.steps)
    out = {"workload": "serving", "dtype": "bf16", "data": "random weights and tokens", "device": torch.cuda.get_device_name(), "peaks": _peaks()[2]}
    kernels = {"ludesun": run_kernels, "lanilix": run_kernels_lanilix, "mabedra": run_kernels_mabedra, "dubazen": run_kernels_dubazen}[args.serving_design]
    out["kernels" if args.kernels else "models"] = kernels(args) if args.kernels else run_models(args)
    if os.environ.get("BENCH_SERVING_OUT"):
        Path(os.environ["BENCH_SERVING_OUT"]).write_text(json.dumps(out, indent=1))
    print(json.dumps({k: v for k, v in out.items() if k not in ("kernels", "models")}), flush=True)
    return 0
