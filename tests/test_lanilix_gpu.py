"""Lanilix kernels and engine paths on the GPU against the plain oracle (tests/lanilix_oracle.py)."""
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(__file__))
import lanilix_oracle as oracle                       # noqa: E402
from lanilix_util import CONFIGS, attn, check, cut, err, feed, layer, make_engine, model, reference, seq   # noqa: E402

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


def rel(a, b):
    a, b = a.detach().cpu().double(), b.double()
    return ((a - b).norm() / b.norm().clamp_min(1e-30)).item()


def batch(lens, starts, slots=None, pages=None):
    """SpanBatch of packed spans, several-token spans first; ``pages`` [span] lists give the paged part."""
    from polyrl_b200.ops.mixers import PAGE, SpanBatch

    n_long = sum(x > 1 for x in lens)
    cu = torch.tensor([0] + lens).cumsum(0).to(torch.int32)
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(starts, lens)])
    seq_of = torch.repeat_interleave(torch.arange(len(lens), dtype=torch.int32), torch.tensor(lens))
    if pages is None:
        table, kv = torch.zeros(len(lens), 1, dtype=torch.int32), torch.zeros_like(pos)
    else:
        width = max(len(p) for p in pages)
        table = torch.tensor([p + [0] * (width - len(p)) for p in pages], dtype=torch.int32)
        kv = table.long()[seq_of.long(), pos // PAGE] * PAGE + pos % PAGE
    return SpanBatch(cu=cu.to(DEV), start=torch.tensor(starts, dtype=torch.int32, device=DEV),
                     slot=torch.tensor(slots or list(range(1, len(lens) + 1)), device=DEV), pos=pos.to(DEV), kv_slot=kv.to(DEV),
                     kv_len=(pos + 1).int().to(DEV), table=table.to(DEV), seq_of=seq_of.to(DEV) if n_long else None, n_long=n_long,
                     t_long=sum(x for x in lens if x > 1), max_long=max(lens) if n_long else 0, max_len=max(s + n for s, n in zip(starts, lens)))


# ---------------------------------------------------------------------------------------------- gated delta rule
SIZES = [(1, 1, 1, 1), (3, 1, 7, 10), (4, 2, 24, 40), (2, 1, 64, 64), (3, 3, 128, 128), (6, 2, 72, 136), (5, 1, 128, 72), (2, 2, 130, 33), (1, 1, 200, 72),
         (2, 1, 300, 40), (1, 1, 512, 32)]


@pytest.mark.parametrize("dtype,chunk_min", [(BF, 2), (BF, 1 << 30), (F32, 0)])
@pytest.mark.parametrize("H,G,N,V", SIZES)
def test_delta_scan(dtype, chunk_min, H, G, N, V, monkeypatch):
    """Every form of the recurrence (tcgen05 chunks, token by token, single step): fresh spans, then a second call that continues some of them
    in other places of the batch; outputs and final states."""
    from polyrl_b200.ops import mixers as M

    monkeypatch.setattr(M, "CHUNK_MIN", chunk_min)
    lens = {"a": 300, "b": 128, "c": 9, "d": 2, "e": 1, "f": 65, "g": 64}
    cuts = {"a": 140, "b": 127, "c": 1, "d": 1, "e": 1, "f": 64, "g": 63}
    g = gen(N + V)
    # keys and queries share a direction (as after silu), decays from almost none to strong, write strengths up to one
    data = {k: dict(q=(torch.randn(n, G * N, generator=g) + 0.7).to(dtype), k=(torch.randn(n, G * N, generator=g) + 0.7).to(dtype),
                    v=torch.randn(n, H * V, generator=g).to(dtype), a=torch.randn(n, H, generator=g) * 2, b=torch.randn(n, H, generator=g) * 3 + 1)
            for k, n in lens.items()}
    bias, a_log, qs = torch.randn(H, generator=g) - 2, torch.linspace(-3, 1.5, H), N ** -0.5
    want, fin = {}, {}
    for k, x in data.items():
        y, n = {m: t.double() for m, t in x.items()}, lens[k]
        decay = torch.exp(-torch.exp(a_log.double()) * oracle.softplus(y["a"] + bias.double()))
        o, S = oracle.delta_scan(oracle.unit(y["q"].reshape(n, G, N)) * qs, oracle.unit(y["k"].reshape(n, G, N)), y["v"].reshape(n, H, V),
                                 torch.sigmoid(y["b"]), decay)
        want[k], fin[k] = o.reshape(n, -1), S
    cache = {"S": torch.full((9, H, N, V), 9.0, device=DEV)}
    slot = {k: i + 1 for i, k in enumerate(lens)}
    got = {k: [] for k in lens}

    def call(part):                     # [(name, lo, hi)]
        part = sorted(part, key=lambda p: p[2] - p[1] == 1)
        b = batch([hi - lo for _, lo, hi in part], [lo for _, lo, _ in part], [slot[k] for k, _, _ in part])
        c = {n: torch.cat([data[k][n][lo:hi] for k, lo, hi in part]).to(DEV) for n in ("q", "k", "v", "a", "b")}
        out = M.scan(M.DELTA, c["q"], c["k"], c["v"], M.Gates(c["a"], c["b"], b0=bias.to(DEV), a_log=a_log.to(DEV)), qs, cache, b)
        for (k, lo, hi), y in zip(part, out.cpu().split([hi - lo for _, lo, hi in part])):
            got[k].append(y)

    call([(k, 0, cuts[k]) for k in lens])
    call([(k, cuts[k], lens[k]) for k in reversed(lens) if cuts[k] < lens[k]])
    M.check_errors(cache["S"].device)
    tol = 6e-3 if dtype == BF else 2e-5
    for k in lens:
        y = torch.cat(got[k])
        assert rel(y, want[k]) < tol, k
        assert rel(y[-1:], want[k][-1:]) < 3 * tol, k
        assert rel(cache["S"][slot[k]], fin[k]) < (2e-4 if dtype == BF else 2e-5), k
    assert (cache["S"][0] == 9).all() and (cache["S"][8] == 9).all()


@pytest.mark.parametrize("case", ["repeat", "no_decay", "strong_decay"])
def test_delta_chunks_with_extreme_keys(case):
    """One key over and over with full writes (the triangular system at its worst), no decay at all, and decays that underflow."""
    from polyrl_b200.ops import mixers as M

    n, N, V = 200, 64, 64
    g = gen(3)
    k = torch.randn(n, N, generator=g)
    if case == "repeat":
        k = k[:1].expand(n, N) + 1e-3 * torch.randn(n, N, generator=g)
    q, v = torch.randn(n, N, generator=g).to(BF), torch.randn(n, V, generator=g).to(BF)
    k = k.to(BF)
    a = torch.full((n, 1), {"repeat": -20.0, "no_decay": -60.0, "strong_decay": 30.0}[case])
    a[::7] -= 25.0 if case == "strong_decay" else 0.0
    b, a_log = torch.full((n, 1), 8.0), torch.tensor([2.0])
    y = [x.double() for x in (q, k, v)]
    decay = torch.exp(-torch.exp(a_log.double()) * oracle.softplus(a.double()))
    want, S = oracle.delta_scan(oracle.unit(y[0])[:, None], oracle.unit(y[1])[:, None], y[2][:, None], torch.sigmoid(b.double()), decay)
    cache = {"S": torch.zeros(2, 1, N, V, device=DEV)}
    out = M.scan(M.DELTA, q.to(DEV), k.to(DEV), v.to(DEV), M.Gates(a.to(DEV), b.to(DEV), a_log=a_log.to(DEV)), 1.0, cache, batch([n], [0]))
    M.check_errors(out.device)
    assert rel(out, want.reshape(n, V)) < 6e-3 and rel(cache["S"][1], S[0]) < 1e-3


# ---------------------------------------------------------------------------------------------- windowed attention
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("H,G,d,rot", [(1, 1, 2, 2), (6, 2, 10, 6), (4, 4, 24, 24), (8, 2, 64, 32), (16, 1, 128, 64), (4, 2, 72, 0), (20, 1, 40, 8), (2, 2, 136, 16)])
def test_windowed_attention(dtype, H, G, d, rot):
    """Norm over the whole projection, pair rotation, cache writes and every attention kernel: a prompt, a portion beside single tokens, single tokens;
    windows and kept tokens at page and tile edges."""
    from polyrl_b200.models.hybrid import cache_width, packs
    from polyrl_b200.ops import mixers as M

    g, eps, scale = gen(d + H), 1e-5, 2.0 * d ** -0.5
    n = {"a": 290, "b": 40, "c": 171}
    p = {k: (torch.randn(m, (H + G) * d, generator=g) * 2).to(dtype) for k, m in n.items()}
    wq, wk = 1 + 0.3 * torch.randn(H * d, generator=g), 1 + 0.3 * torch.randn(G * d, generator=g)
    width = cache_width(dict(dim=d), dtype)
    freq = M.rope_frequencies(rot, 200.0, DEV)
    pages = {"a": list(range(30, 49)), "b": [3, 1, 2], "c": list(range(20, 9, -1))}
    q_, k_, v_ = {}, {}, {}
    for k, x in p.items():
        x, pos = x.double(), torch.arange(n[k])
        raw = x[:, H * d:]
        q_[k] = oracle.rotate_pairs((oracle.rms(x[:, :H * d], eps) * wq.double()).reshape(-1, H, d), pos, 200.0, rot)
        k_[k] = oracle.rotate_pairs((oracle.rms(raw, eps) * wk.double()).reshape(-1, G, d), pos, 200.0, rot)
        v_[k] = raw.reshape(-1, G, d)
    tol = 1.5e-2 if dtype == BF else 2e-5
    for window, keep in [(16, 0), (17, 3), (128, 16), (129, 17), (1, 1), (100, 130), (1000, 4)]:
        want = {k: oracle.window_attention(q_[k], k_[k], v_[k], scale, window, keep) for k in n}
        kp, vp = (torch.full((50, G, M.PAGE, width), 7.0, device=DEV, dtype=dtype) for _ in range(2))
        got = {k: [] for k in n}

        def call(part):
            part = sorted(part, key=lambda x: x[2] - x[1] == 1)
            b = batch([hi - lo for _, lo, hi in part], [lo for _, lo, _ in part], pages=[pages[k] for k, _, _ in part])
            x = torch.cat([p[k][lo:hi] for k, lo, hi in part]).to(DEV)
            tl = b.t_long if packs(dict(dim=d), dtype, True) else 0
            behind = any(lo > 0 for _, lo, hi in part if hi - lo > 1)
            q, kv = M.qk_prep(x, H, d, wq.to(DEV), wk.to(DEV), freq, kp, vp, b, eps, tl > 0 and not behind)
            outs = []
            if tl:
                if behind:              # the keys that some token of a portion sees: kept ones, then the window of its first token
                    idx, cu = [], [0]
                    for k, lo, hi in part[:b.n_long]:
                        js = [j for j in range(hi) if j < keep or j > lo - window]
                        idx += [pages[k][j // 16] * 16 + j % 16 for j in js]
                        cu.append(len(idx))
                    kk, vv = M.gather_keys(kp, vp, torch.tensor(idx, device=DEV))
                    cu_k = torch.tensor(cu, dtype=torch.int32, device=DEV)
                else:
                    kk, vv, cu_k = kv[0][:tl], kv[1][:tl], b.cu[:b.n_long + 1]
                outs.append(M.window_attention_varlen(q[:tl], kk, vv, b.cu[:b.n_long + 1], cu_k, scale, window, keep))
            if tl < b.tokens:
                lo = b.n_long if tl else 0
                outs.append(M.window_attention(q[tl:], kp, vp, b.table[lo:], None if b.seq_of is None or tl else b.seq_of[tl:], b.kv_len[tl:], scale, window,
                                               keep, b.max_len))
            o = torch.cat(outs)
            assert (o[..., d:] == 0).all()
            for (k, lo, hi), y in zip(part, o[..., :d].cpu().split([hi - lo for _, lo, hi in part])):
                got[k].append(y)

        call([("a", 0, 150), ("b", 0, 2), ("c", 0, 1)])
        call([("a", 150, 287), ("b", 2, 3), ("c", 1, 170)])
        for i in range(3):
            call([("a", 287 + i, 288 + i), ("b", 3 + i, 4 + i)] + ([("c", 170, 171)] if i == 1 else []))
        for k in n:
            y = torch.cat(got[k])
            d_ = (y.double() - want[k][:len(y)]).pow(2).mean(-1).sqrt()           # per position and head
            e = (d_ / want[k].pow(2).mean().sqrt()).max().item()
            assert e < (0.1 if dtype == BF else 5e-5) and rel(y, want[k][:len(y)]) < tol, (window, keep, k, e)


def test_paged_decode_without_a_window_is_unchanged():
    from polyrl_b200 import ops

    g = gen(1)
    q, kc, vc = (torch.randn(*s, generator=g).to(DEV, BF) for s in ((3, 8 * 128), (20, 2, 16, 128), (20, 2, 16, 128)))
    bt = torch.randperm(18, generator=g).reshape(3, 6).int().to(DEV)
    sl = torch.tensor([90, 1, 33], dtype=torch.int32, device=DEV)
    a = ops.paged_decode_attention(q, kc, vc, bt, sl, 8, 2, 128, 0.09)
    for splits in (1, 3):
        assert rel(ops.paged_decode_attention(q, kc, vc, bt, sl, 8, 2, 128, 0.09, splits=splits, window=96), a.cpu().double()) < 5e-3
    from polyrl_b200.ops import reference as ref

    want = ref.paged_decode_attention(q.cpu().float(), kc.cpu().float(), vc.cpu().float(), bt.cpu(), sl.cpu(), 8, 2, 128, 0.09)
    assert rel(a, want.double()) < 1e-2


# ---------------------------------------------------------------------------------------------- rows and feed-forward
@pytest.mark.parametrize("M_,F,K", [(1, 128, 64), (5, 384, 104), (128, 256, 256), (129, 1024, 128), (300, 128, 64), (3, 40, 37), (200, 45, 24)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_clamped_glu(dtype, M_, F, K):
    from polyrl_b200.ops import mixers as M
    from polyrl_b200.ops import reference as ref

    g = gen(M_ + F)
    x, wg, wu = torch.randn(M_, K, generator=g).to(dtype), torch.randn(F, K, generator=g).to(dtype), torch.randn(F, K, generator=g).to(dtype)
    wg, wu = wg * (2 * K ** -0.5), wu * (2 * K ** -0.5)
    w = ref.interleave_gate_up(wg, wu) if F % 128 == 0 else torch.cat([wg, wu])
    got = M.linear_clamped_glu(x.to(DEV), w.to(DEV), 1.3, 1.702)
    want = oracle.clamped_glu(x.double(), wg.double(), wu.double(), torch.eye(F, dtype=oracle.D), 1.3)
    assert rel(got, want) < (6e-3 if dtype == BF else 2e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("W,groups", [(37, 1), (96, 4), (60, 5), (4096, 32), (1024, 8)])
def test_rows(dtype, W, groups):
    from polyrl_b200.ops import mixers as M

    g = gen(W)
    emb, w = torch.randn(11, W, generator=g).to(dtype), 1 + 0.2 * torch.randn(W, generator=g)
    ids = torch.tensor([3, 0, 10, 3])
    x, h = M.embed(ids.to(DEV), emb.to(DEV), w.to(DEV), 1e-5)
    tol = 4e-3 if dtype == BF else 1e-6
    assert torch.equal(x.cpu(), emb[ids].float()) and rel(h, oracle.rms(emb[ids].double(), 1e-5) * w.double()) < tol
    y, z = torch.randn(9, W, generator=g).to(dtype), torch.randn(9, 2 * W, generator=g).to(dtype)
    got = M.gated_norm(y.to(DEV), z.to(DEV)[:, W:], w.to(DEV), groups, 1e-5, M.SILU_LAST)
    want = oracle.rms(y.double().reshape(9, groups, -1), 1e-5).reshape(9, W) * w.double() * oracle.silu(z[:, W:].double())
    assert rel(got, want) < tol


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("ch,taps", [(5, 3), (64, 4), (136, 2), (24, 1), (40, 6)])
def test_short_convolution_without_bias(dtype, ch, taps):
    from polyrl_b200.ops import mixers as M

    g = gen(ch + taps)
    n = {"a": 40, "b": 21, "c": 3, "d": 1}
    x = {k: torch.randn(m, ch, generator=g).to(dtype) for k, m in n.items()}
    w = torch.randn(ch, taps, generator=g)
    state = torch.full((6, taps - 1, ch), 5.0, device=DEV, dtype=dtype)
    got = {k: [] for k in n}
    for part in ([("a", 0, 17), ("b", 0, 2), ("c", 0, 1), ("d", 0, 1)], [("a", 17, 18), ("b", 2, 3), ("c", 1, 2)], [("a", 18, 40), ("b", 3, 21), ("c", 2, 3)]):
        b = batch([hi - lo for _, lo, hi in part], [lo for _, lo, _ in part], [list(n).index(k) + 1 for k, _, _ in part])
        out = M.conv_silu(torch.cat([x[k][lo:hi] for k, lo, hi in part]).to(DEV), w.t().contiguous().to(DEV), None, state, b)
        for (k, lo, hi), y in zip(part, out.cpu().split([hi - lo for _, lo, hi in part])):
            got[k].append(y)
    for k in n:
        assert rel(torch.cat(got[k]), oracle.short_conv(x[k].double(), w.double())) < (4e-3 if dtype == BF else 1e-6), k


# ---------------------------------------------------------------------------------------------- the engine
REAL = model(256, 300, layer("delta", dict(heads=4, kv_heads=2, dim=128, vdim=128, conv=4), 384), layer("attention", attn(8, 2, 128, 100, 5, 64), 256),
             layer("delta", dict(heads=2, kv_heads=2, dim=64, vdim=64, conv=2)), layer("attention", attn(4, 1, 64, 33, 2, 64), 256, 0.8),
             layer("delta", dict(heads=4, kv_heads=2, dim=128, vdim=128, conv=4), 384, weights_of=0))
WIDE = model(96, 120, layer("delta", dict(heads=2, kv_heads=1, dim=136, vdim=48, conv=4), 64), layer("attention", attn(2, 1, 144, 40, 3, 80), 72),
             layer("attention", attn(34, 2, 16, 50, 1, 8)))
ALL = {**CONFIGS, "real": REAL, "wide": WIDE}


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg in ALL.items():
        sd = oracle.random_model(cfg, seed=len(name))
        d = tmp_path_factory.mktemp("m") / name
        oracle.write_model(cfg, sd, d)
        toks = {"a": seq(230, cfg["vocab"], 1), "b": seq(67, cfg["vocab"], 2), "c": seq(1, cfg["vocab"], 3), "d": seq(90, cfg["vocab"], 4)}
        out[name] = (cfg, sd, d, toks, reference(cfg, sd, toks))
    return out


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", ["odd", "even", "real", "wide"])
def test_engine_schedules(folders, name, dtype):
    """Whole prompts, token by token, portions of several sizes, and mixed batches over pages and slots that are used again."""
    cfg, sd, d, toks, want = folders[name]
    eng = make_engine(d, DEV, dtype, max_len=256, tokens=640)
    runs = {"whole": [[(k, len(t))] for k, t in toks.items()],
            "decode": [[("a", 150)]] + [[("a", 1)]] * 80,
            "portions": [[("a", x)] for x in cut(230, (2, 17, 64, 3, 65))],
            "mixed": [[("b", 29), ("a", 2), ("c", 1)], [("a", 131), ("b", 1), ("d", 16)], [("d", 1), ("a", 1), ("b", 2)], [("b", 35), ("d", 3), ("a", 96)],
                      [("d", 70)]]}
    for what, steps in runs.items():
        part = {k: t for k, t in toks.items() if any(k == e[0] for st in steps for e in st)}
        got = feed(eng, part, steps)
        for k in part:
            check(got[k], want[k], dtype, (what, k))
    assert not eng.running


def test_sizes_of_one(folders):
    cfg, sd, d, toks, want = folders["one"]
    for dtype in (F32, BF):
        eng = make_engine(d, DEV, dtype, max_len=256)
        for steps in ([[("a", 230)]], [[("a", 100)]] + [[("a", 1)]] * 30 + [[("a", 100)]]):
            check(feed(eng, {"a": toks["a"]}, steps)["a"], want["a"], dtype)


def test_batch_portions_and_slots_do_not_matter(folders):
    """The logits of a request alone, cut differently, and among others on other pages agree to rounding (bf16 kernels)."""
    cfg, sd, d, toks, want = folders["real"]
    eng = make_engine(d, DEV, BF, max_len=256, tokens=640)
    base = feed(eng, {"a": toks["a"]}, [[("a", 230)]])["a"]
    others = [feed(eng, {"a": toks["a"]}, [[("a", x)] for x in cut(230, (33, 2, 70))])["a"],
              feed(eng, {k: toks[k] for k in "abd"}, [[("b", 67), ("a", 65)], [("d", 88), ("a", 100)], [("a", 65), ("d", 2)]])["a"]]
    for o in others:
        e = ((o - base).pow(2).mean(-1).sqrt() / base.pow(2).mean().sqrt())
        assert e.median() < 0.02 and e.max() < 0.3


def test_long_decoding(folders):
    cfg, sd, d, toks, want = folders["real"]
    check(feed(make_engine(d, DEV, BF, max_len=256), {"a": toks["a"]}, [[("a", 2)]] + [[("a", 1)]] * 228)["a"], want["a"], BF)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_greedy_generation(folders, dtype):
    from test_lanilix_cpu import greedy_oracle

    cfg, sd, d, _, _ = folders["even"]
    eng = make_engine(d, DEV, dtype, max_len=128)
    prompts = [seq(n, cfg["vocab"], n) for n in (5, 1, 40, 23, 30, 9)]
    reqs = eng.generate(prompts, dict(max_new_tokens=24, temperature=0.0))
    for p, (r,) in zip(prompts, reqs):
        if dtype == F32:
            assert r.output_ids == greedy_oracle(cfg, sd, p, 24)
        else:       # a near tie may fall the other way: every token is close to the best of its own prefix
            lg = oracle.forward(cfg, sd, p + r.output_ids)[len(p) - 1:-1]
            gap = lg.max(-1).values - lg.gather(1, torch.tensor(r.output_ids)[:, None])[:, 0]
            assert len(r.output_ids) == 24 and gap.max() < 0.15 * lg.std()


def test_weight_update_reaches_captured_graphs(folders, tmp_path):
    cfg, _, d, toks, _ = folders["even"]
    eng = make_engine(d, DEV, F32, max_len=128)
    t = {"b": toks["b"]}
    steps = [[("b", 60)]] + [[("b", 1)]] * 7
    feed(eng, t, steps)
    sd = oracle.random_model(cfg, 77)
    oracle.write_model(cfg, sd, tmp_path / "n")
    other = make_engine(tmp_path / "n", DEV, F32, max_len=128)
    eng.set_weights(other.embed_w, [dict(w) for w in _stored(tmp_path / "n", cfg)], _head(tmp_path / "n"))
    assert err(feed(eng, t, steps)["b"], reference(cfg, sd, t)["b"]) < 1e-4


def _stored(folder, cfg):
    return _weights(folder).layers


def _head(folder):
    return _weights(folder).head


def _weights(folder):
    from polyrl_b200.models import TransformerWeights, get_model_config
    from polyrl_b200.models.hf_io import load_state_dict

    c = get_model_config(str(folder))
    w = TransformerWeights(c, device=DEV, dtype=F32, init=False)
    w.load_state_dict({k: v.to(DEV, F32) for k, v in load_state_dict(c, folder).items()})
    return w
