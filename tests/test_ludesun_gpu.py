"""Ludesun kernels and engine paths on the GPU against the plain oracle (tests/ludesun_oracle.py)."""
import os
import sys

import pytest
import torch
import torch.nn.functional as F

sys.path.insert(0, os.path.dirname(__file__))
import ludesun_oracle as oracle                       # noqa: E402
from ludesun_util import CONFIGS, check, cut, err, feed, layer, make_engine, model, reference, seq   # noqa: E402
from test_ludesun_cpu import far_model, greedy_oracle                                          # noqa: E402

pytestmark = pytest.mark.gpu
DEV = "cuda"


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


def rel(a, b):
    a, b = a.detach().cpu().double(), b.double()
    return ((a - b).norm() / b.norm().clamp_min(1e-30)).item()


def spans(lens, starts, slots=None):
    """SpanBatch of packed spans (several-token spans first), without the paged part."""
    from polyrl_b200.ops.mixers import SpanBatch

    n_long = sum(x > 1 for x in lens)
    cu = torch.tensor([0] + list(torch.tensor(lens).cumsum(0)), dtype=torch.int32)
    t = int(cu[-1])
    seq_of = torch.repeat_interleave(torch.arange(len(lens), dtype=torch.int32), torch.tensor(lens))
    z = torch.zeros(t, dtype=torch.long, device=DEV)
    return SpanBatch(cu=cu.to(DEV), start=torch.tensor(starts, dtype=torch.int32, device=DEV),
                     slot=torch.tensor(slots or list(range(1, len(lens) + 1)), device=DEV), pos=z, kv_slot=z, kv_len=z.int(),
                     table=torch.zeros(len(lens), 1, dtype=torch.int32, device=DEV), seq_of=seq_of.to(DEV) if n_long else None, n_long=n_long,
                     t_long=sum(x for x in lens if x > 1), max_long=max(lens) if n_long else 0)


# ---------------------------------------------------------------------------------------------- recurrences
SIZES = [(1, 1, 1, 1), (3, 1, 7, 10), (2, 2, 24, 40), (4, 2, 64, 64), (2, 1, 128, 64), (3, 3, 72, 96), (2, 2, 130, 33), (1, 1, 200, 72), (2, 2, 256, 128),
         (1, 1, 300, 40), (2, 1, 512, 32)]


@pytest.mark.parametrize("mode", ["ssd", "mlstm"])
@pytest.mark.parametrize("dtype,tc_min", [(torch.bfloat16, 2), (torch.bfloat16, 1 << 30), (torch.float32, 0)])
@pytest.mark.parametrize("H,G,N,V", SIZES)
def test_scan(mode, dtype, tc_min, H, G, N, V, monkeypatch):
    """Every form of the recurrence kernels (tcgen05 chunks, mma chunks, token by token, single step).  Fresh spans, then a second call that continues some of them in other places of the batch: outputs and final states."""
    from polyrl_b200.ops import mixers as M

    monkeypatch.setattr(M, "TC_MIN", tc_min)
    if mode == "mlstm":
        G = H
    lens = {"a": 300, "b": 128, "c": 9, "d": 2, "e": 1, "f": 129}
    cuts = {"a": 140, "b": 127, "c": 1, "d": 1, "e": 1, "f": 128}
    g = gen(N + V)
    data = {k: dict(q=torch.randn(n, G * N, generator=g).to(dtype), k=(torch.randn(n, G * N, generator=g) * N ** -0.5).to(dtype),
                    v=torch.randn(n, H * V, generator=g).to(dtype), g0=torch.randn(n, H, generator=g) * 2, g1=torch.randn(n, H, generator=g) + 1)
            for k, n in lens.items()}
    b0, b1 = torch.randn(H, generator=g), torch.randn(H, generator=g) + 2
    a_log, dskip = torch.linspace(-2.5, 0.5, H), torch.randn(H, generator=g)
    if mode == "mlstm":                 # small input gates: the running maximum comes from the forget path and the floor
        b0[0] -= 4
    cap, qs = 7.0, N ** -0.5
    want, state = {}, {}
    for k, x in data.items():
        y = {n: t.double() for n, t in x.items()}
        n = lens[k]
        if mode == "ssd":
            dt = F.softplus(y["g0"] + b0.double())
            want[k] = oracle.mamba2_scan(y["v"].reshape(n, H, V), y["k"].reshape(n, G, N), y["q"].reshape(n, G, N) * qs, dt, a_log.double(),
                                         dskip.double()).reshape(n, -1)
        else:
            i = cap * torch.tanh((y["g0"] + b0.double()) / cap)
            f = F.logsigmoid(cap * torch.tanh((y["g1"] + b1.double()) / cap))
            want[k] = oracle.mlstm_scan(y["q"].reshape(n, H, N) * qs, y["k"].reshape(n, H, N), y["v"].reshape(n, H, V), i, f).reshape(n, -1)
    f32 = dict(device=DEV, dtype=torch.float32)
    cache = {"S": torch.full((8, H, N, V), 9.0, **f32), "n": torch.full((8, H, N), 9.0, **f32), "m": torch.full((8, H), 9.0, **f32)}
    slot = {k: i + 1 for i, k in enumerate(lens)}
    got = {k: [] for k in lens}

    def call(part):                     # [(name, lo, hi)]
        part = sorted(part, key=lambda p: p[2] - p[1] == 1)
        b = spans([hi - lo for _, lo, hi in part], [lo for _, lo, _ in part], [slot[k] for k, _, _ in part])
        c = {n: torch.cat([data[k][n][lo:hi] for k, lo, hi in part]).to(DEV) for n in ("q", "k", "v", "g0", "g1")}
        gates = M.Gates(c["g0"], c["g1"], b0.to(DEV), b1.to(DEV), a_log.to(DEV), dskip.to(DEV), cap)
        out = M.scan(M.SSD if mode == "ssd" else M.MLSTM, c["q"], c["k"], c["v"], gates, qs, cache, b)
        for (k, lo, hi), y in zip(part, out.cpu().split([hi - lo for _, lo, hi in part])):
            got[k].append(y)

    call([(k, 0, cuts[k]) for k in lens])
    call([(k, cuts[k], lens[k]) for k in reversed(lens) if cuts[k] < lens[k]])
    tol = 6e-3 if dtype == torch.bfloat16 else 2e-5
    for k in lens:
        y = torch.cat(got[k])
        assert rel(y, want[k]) < tol, k
        assert rel(y[-1:], want[k][-1:]) < 3 * tol, k
    M.check_errors(cache["S"].device)
    # the state itself
    fin = {k: cache["S"][slot[k]].cpu().double() for k in lens}
    for k in ("a", "f"):
        x = {n: t.double() for n, t in data[k].items()}
        S = torch.zeros(H, N, V, dtype=oracle.D)
        m = torch.zeros(H, dtype=oracle.D)
        for t in range(lens[k]):
            kt = x["k"][t].reshape(G, N).repeat_interleave(H // G, 0)
            if mode == "ssd":
                add = F.softplus(x["g0"][t] + b0.double())
                keep = torch.exp(-torch.exp(a_log.double()) * add)
            else:
                i = cap * torch.tanh((x["g0"][t] + b0.double()) / cap)
                f = F.logsigmoid(cap * torch.tanh((x["g1"][t] + b1.double()) / cap))
                m2 = torch.maximum(f + m, i)
                keep, add, m = torch.exp(f + m - m2), torch.exp(i - m2), m2
            S = keep[:, None, None] * S + (add[:, None] * kt)[:, :, None] * x["v"][t].reshape(H, 1, V)
        assert rel(fin[k], S) < (3e-5 if dtype == torch.bfloat16 else 1e-5), k


# ---------------------------------------------------------------------------------------------- convolution, norms, GELU
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("ch,taps", [(5, 4), (64, 4), (136, 2), (24, 1), (1040, 5)])
def test_conv(dtype, ch, taps):
    from polyrl_b200.ops import mixers as M

    g = gen(ch)
    x = {k: torch.randn(n, ch, generator=g).to(dtype) for k, n in dict(a=40, b=7, c=2, d=3).items()}
    w, bias = torch.randn(ch, taps, generator=g), torch.randn(ch, generator=g)
    state = torch.full((6, taps - 1, ch), 5.0, dtype=dtype, device=DEV)
    got = {k: [] for k in x}
    for part in ([("a", 0, 11), ("b", 0, 2), ("c", 0, 1), ("d", 0, 1)], [("a", 11, 13), ("b", 2, 3), ("c", 1, 2), ("d", 1, 2)],
                 [("b", 3, 4), ("a", 13, 14), ("d", 2, 3)], [("b", 4, 7), ("a", 14, 40)]):
        b = spans([hi - lo for _, lo, hi in part], [lo for _, lo, _ in part], ["abcd".index(k) + 1 for k, _, _ in part])
        wide = torch.cat([x[k][lo:hi] for k, lo, hi in part]).to(DEV)
        wide = F.pad(wide, (8, 8))[:, 8:8 + ch]                                    # a column slice of a wider projection
        y = M.conv_silu(wide, w.t().contiguous().to(DEV), bias.to(DEV), state, b)
        for (k, lo, hi), p in zip(part, y.cpu().split([hi - lo for _, lo, hi in part])):
            got[k].append(p)
    for k in x:
        want = oracle.silu(oracle.causal_conv(x[k].double(), w.double(), bias.double()))
        assert rel(torch.cat(got[k]), want) < (4e-3 if dtype == torch.bfloat16 else 1e-6), k


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("W,groups", [(37, 1), (96, 4), (60, 5), (4096, 8), (8192, 2), (512, 512)])
def test_norms(dtype, W, groups):
    from polyrl_b200.ops import mixers as M

    g = gen(W)
    y, z = (torch.randn(9, W, generator=g) * 3).to(dtype), torch.randn(9, W, generator=g).to(dtype)
    w, w2 = torch.randn(W, generator=g), torch.randn(W, generator=g)
    tol = 4e-3 if dtype == torch.bfloat16 else 1e-6
    yd, zd, wd = y.double(), z.double(), w.double()
    for first in (True, False):
        got = M.gated_norm(y.to(DEV), z.to(DEV), w.to(DEV), groups, 1e-3, first)
        want = oracle.grouped_rms(yd * oracle.silu(zd), groups, 1e-3) * wd if first else oracle.grouped_rms(yd, groups, 1e-3) * wd * torch.sigmoid(zd)
        assert rel(got, want) < tol
    x = torch.randn(9, W, generator=g)
    xd = x.double() + oracle.rms(yd, 1e-3) * wd
    for nxt in (None, w2):
        xg = x.to(DEV)
        h = M.norm_add_(y.to(DEV), xg, w.to(DEV), 1e-3, None if nxt is None else nxt.to(DEV))
        assert rel(xg, xd) < 1e-6
        assert rel(h, xd if nxt is None else oracle.rms(xd, 1e-3) * w2.double()) < tol
    assert rel(M.rms(x.to(DEV), w.to(DEV), 1e-3, dtype), oracle.rms(x.double(), 1e-3) * wd) < tol


@pytest.mark.parametrize("M_,N,K", [(1, 72, 64), (5, 320, 104), (128, 256, 256), (129, 1000, 128), (300, 128, 64), (700, 512, 328)])
def test_gelu_gemm(M_, N, K):
    from polyrl_b200.ops import mixers as M

    x, w = torch.randn(M_, K, generator=gen(1)).bfloat16(), (torch.randn(N, K, generator=gen(2)) * 2 * K ** -0.5).bfloat16()
    want = oracle.gelu_tanh(x.double() @ w.double().T)
    assert rel(M.linear_gelu(x.to(DEV), w.to(DEV)), want) < 4e-3
    assert rel(M.linear_gelu(x.float().to(DEV), w.float().to(DEV)), want) < 1e-6
    odd = w[:N - 3]                                            # rows not a multiple of 8
    assert rel(M.linear_gelu(x.to(DEV), odd.to(DEV)), want[:, :N - 3]) < 6e-3


# ---------------------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])
@pytest.mark.parametrize("H,r,rd,d", [(1, 3, 2, 1), (2, 13, 4, 6), (4, 64, 16, 32), (20, 128, 64, 24), (5, 96, 8, 8), (40, 512, 64, 128), (3, 272, 32, 16)])
def test_paged_latent_attention(dtype, H, r, rd, d):
    """Every row against plain attention over the same cache rows: page borders, one key that stands out, idle rows, splits."""
    from polyrl_b200.ops import ext
    from polyrl_b200.ops import mixers as M

    g = gen(r)
    lens = [1, 2, 15, 16, 17, 31, 32, 33, 64, 0, 257, 700]
    R, width = len(lens), 44
    perm = torch.randperm(R * width, generator=g) + 1
    table = perm.reshape(R, width).int()
    pool = torch.randn(R * width + 1, 1, 16, r + rd, generator=g).to(dtype)
    q_lat = torch.randn(H, R, r, generator=g).to(dtype)
    q = torch.randn(R, H, d + rd + 3, generator=g).to(dtype)
    scale = 2.0 * (r + rd) ** -0.5
    for i, n in enumerate(lens):                               # one key of every row answers its query: place it at an edge
        if n:
            j = [0, n - 1, n // 2, min(n - 1, 15), min(n - 1, 16)][i % 5]
            pool[table[i, j // 16].long(), 0, j % 16, :r] = (q_lat[i % H, i].float() * 3).to(dtype)
    sink = torch.randn(H, generator=g) * 3
    want = torch.zeros(H, R, r, dtype=oracle.D)
    for i, n in enumerate(lens):
        kv = pool[table[i].long(), 0].reshape(-1, r + rd)[:n].double()
        qq = torch.cat([q_lat[:, i], q[i, :, d:d + rd]], -1).double()
        for h in range(H if n else 0):
            s = kv @ qq[h] * scale
            e = torch.exp(s - s.max())
            want[h, i] = (e @ kv[:, :r]) / (e.sum() + torch.exp(sink[h].double() - s.max()))
    args = (q_lat.to(DEV), q.to(DEV), d, pool.to(DEV), table.to(DEV), None, torch.tensor(lens, dtype=torch.int32, device=DEV), sink.to(DEV), scale)
    tol = 6e-3 if dtype == torch.bfloat16 else 1e-5
    outs = [M.latent_attention(*args, 700)]
    C = ext()
    outs.append(C.mix_latent(*args, 1, False))                 # one CTA per (row, head)
    if dtype == torch.bfloat16 and C.mix_latent_tc_ok(r, rd):
        outs += [C.mix_latent(*args, s, True) for s in (1, 2, 5)]
    for o in outs:
        assert rel(o, want) < tol
        for i, n in enumerate(lens):
            assert o[:, i].abs().max().item() == 0 if n == 0 else rel(o[:, i], want[:, i]) < 3 * tol, (i, n)


@pytest.mark.parametrize("dk", [128, 192])
def test_packed_attention_with_sink(dk):
    from polyrl_b200.ops import mixers as M

    g = gen(dk)
    H, lq, lk = 3, [130, 1, 2, 200], [130, 40, 300, 456]
    q = torch.randn(sum(lq), H, dk, generator=g).bfloat16()
    k, v = torch.randn(sum(lk), H, dk, generator=g).bfloat16(), torch.randn(sum(lk), H, 128, generator=g).bfloat16()
    sink = torch.tensor([-2.0, 3.0, 9.0])
    cu = lambda x: torch.tensor([0] + list(torch.tensor(x).cumsum(0)), dtype=torch.int32)
    cq, ck = cu(lq), cu(lk)
    scale = dk ** -0.5
    for i, n in enumerate(lk):
        k[ck[i] + n // 3] = q[cq[i + 1] - 1] * 2               # the last query's key is far back
    got = M.sink_attention_varlen(q.to(DEV), k.to(DEV), v.to(DEV), cq.to(DEV), ck.to(DEV), scale, sink.to(DEV)).cpu().double()
    plain = M.sink_attention_varlen(q.to(DEV), k.to(DEV), v.to(DEV), cq.to(DEV), ck.to(DEV), scale, None).cpu().double()
    for i in range(4):
        qq, kk, vv = q[cq[i]:cq[i + 1]].double(), k[ck[i]:ck[i + 1]].double(), v[ck[i]:ck[i + 1]].double()
        off = lk[i] - lq[i]
        pad = torch.zeros(off, H, dk, dtype=oracle.D)
        for s, o in ((sink.double(), got), (torch.full((H,), -1e9, dtype=oracle.D), plain)):
            want = oracle.sink_attention(torch.cat([pad, qq]), kk, vv, scale, s)[off:]
            assert rel(o[cq[i]:cq[i + 1]], want) < 6e-3
            assert rel(o[cq[i + 1] - 1], want[-1]) < 1.5e-2


# ---------------------------------------------------------------------------------------------- engine
@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    real = model(256, 200, layer("latent_attention", dict(heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=128, q_rank=96, scale=0.072,
                                                          rot=dict(base=10000.0, dims=64)), 520),
                 layer("mamba2", dict(heads=4, vdim=64, state=128, groups=1, conv=4, norm_groups=2), 264),
                 layer("mlstm", dict(heads=2, dim=128, vdim=256, gate_cap=15.0), 256), layer("latent_attention", dict(
                     heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=128, q_rank=96, scale=0.072, rot=dict(base=10000.0, dims=64)), 520, weights_of=0))
    wide = model(96, 70, layer("latent_attention", dict(heads=2, dim=160, rot_dim=48, vdim=136, kv_rank=64, q_rank=32, scale=0.07,
                                                        rot=dict(base=100.0, dims=48)), 64))
    out = {}
    for name, cfg in {**CONFIGS, "real": real, "wide": wide}.items():
        sd = oracle.random_model(cfg, seed=len(name))
        d = tmp_path_factory.mktemp("g") / name
        oracle.write_model(cfg, sd, d)
        out[name] = (cfg, sd, d)
    return out


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", ["odd", "even", "real", "wide"])
def test_engine_schedules(folders, name, dtype):
    """Whole prompts, portions, token by token (the decode graph), unequal batches with pages and slots used again."""
    cfg, sd, d = folders[name]
    v = cfg["vocab"]
    toks = {"a": seq(130, v, 1), "b": seq(33, v, 2), "c": seq(1, v, 3), "d": seq(90, v, 4), "e": seq(20, v, 5)}
    want = reference(cfg, sd, toks)
    eng = make_engine(d, DEV, dtype, tokens=384)
    plans = [[[(k, len(t))] for k, t in toks.items()],
             [[(k, n)] for k, t in toks.items() for n in cut(len(t), (17, 2, 64, 1, 3))],
             [[("d", 40)]] + [[("d", 1)]] * 50 + [[("a", 64)], [("a", 66)], [("b", 33)], [("c", 1)], [("e", 20)]],
             [[("a", 65), ("b", 2), ("c", 1)], [("b", 1), ("a", 2), ("d", 17)], [("b", 1), ("d", 1)], [("b", 29), ("d", 30), ("a", 1)],
              [("e", 2), ("a", 1), ("d", 1)], [("e", 1), ("a", 1), ("d", 1)], [("e", 16), ("d", 39), ("a", 60)], [("e", 1), ("d", 1)]]]
    for plan in plans:
        got = feed(eng, toks, plan)
        for k in toks:
            if k != "c" or dtype == torch.float32:             # (one position is no statistic)
                check(got[k], want[k], dtype, (k, plan[0]))
    assert len(eng.state.free) == 4


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-4), (torch.bfloat16, 0.05)])
def test_far_keys_and_page_borders(tmp_path, dtype, tol):
    for sink in (-3.0, 4.0):
        cfg, sd = far_model(sink)
        oracle.write_model(cfg, sd, tmp_path / f"m{sink}")
        eng = make_engine(tmp_path / f"m{sink}", DEV, dtype)
        for at in (0, 15, 16, 47):
            t = [x + 3 for x in seq(100, 9, at)]
            t[at] = 2
            for q in (at + 1, 64, 80, 99):
                t[q] = 1
            want = oracle.forward(cfg, sd, t)
            for steps in ([100], cut(100, (33, 16, 1)), [60] + [1] * 40):
                assert err(feed(eng, {"a": t}, [[("a", n)] for n in steps])["a"], want) < tol, (at, steps)


def test_long_decoding(folders):
    cfg, sd, d = folders["even"]
    t = seq(400, cfg["vocab"], 9)
    want = oracle.forward(cfg, sd, t)
    for dtype in (torch.float32, torch.bfloat16):
        got = feed(make_engine(d, DEV, dtype, max_len=512), {"a": t}, [[("a", 5)]] + [[("a", 1)]] * 395)
        check(got["a"], want, dtype)


def test_sizes_of_one(folders):
    cfg, sd, d = folders["one"]
    toks = {"a": seq(70, cfg["vocab"], 1)}
    want = reference(cfg, sd, toks)["a"]
    for plan in ([70], [1] * 70, cut(70, (2, 9, 1))):
        check(feed(make_engine(d, DEV, torch.float32), toks, [[("a", n)] for n in plan])["a"], want, torch.float32)


def test_greedy_generation(folders):
    """The engine's own entry point: admission, prefill chunks, decode graphs, slot compaction and reuse."""
    cfg, sd, d = folders["odd"]
    prompts = [seq(n, cfg["vocab"], n) for n in (1, 5, 16, 23, 9, 2, 30)]
    want = [greedy_oracle(cfg, sd, p, 10) for p in prompts]
    for chunk in (16384, 7):
        eng = make_engine(d, DEV, torch.float32, seqs=3, max_len=64, max_prefill_tokens=chunk)
        for _ in range(2):
            out = eng.generate(prompts, dict(max_new_tokens=10, temperature=0.0))
            assert [g[0].output_ids for g in out] == want
    out = make_engine(d, DEV, torch.float32, max_len=64).generate([prompts[3]], dict(max_new_tokens=10, temperature=0.0, n=3))
    assert [r.output_ids for r in out[0]] == [want[3]] * 3
    bf = make_engine(d, DEV, torch.bfloat16, seqs=3, max_len=64).generate(prompts, dict(max_new_tokens=10, temperature=0.0))
    assert all(len(g[0].output_ids) == 10 for g in bf)


def test_weight_update_reaches_captured_graphs(folders):
    from polyrl_b200.models import TransformerWeights
    from polyrl_b200.models.hf_io import load_state_dict

    cfg, sd, d = folders["even"]
    eng = make_engine(d, DEV, torch.float32, max_len=64)
    t = {"a": seq(20, cfg["vocab"], 1)}
    plan = [[("a", 4)]] + [[("a", 1)]] * 16
    feed(eng, t, plan)
    sd2 = oracle.random_model(cfg, seed=77)
    oracle.write_model(cfg, sd2, d.parent / "second")
    w = TransformerWeights(eng.cfg, device=DEV, dtype=torch.float32, init=False)
    w.load_state_dict({k: x.to(DEV, torch.float32) for k, x in load_state_dict(eng.cfg, d.parent / "second").items()})
    eng.set_weights(w.embed, w.layers, w.head)
    assert err(feed(eng, t, plan)["a"], oracle.forward(cfg, sd2, t["a"])) < 1e-4
