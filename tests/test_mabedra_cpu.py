"""Mabedra stacks through the framework's configuration, loader, scheduler, cache / state manager and step functions, on CPU in fp32,
against the plain oracle (tests/mabedra_oracle.py)."""
import io
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(__file__))
import mabedra_oracle as oracle                       # noqa: E402
from mabedra_util import A_EVEN, A_ODD, CONFIGS, attn, cut, dense, err, feed, layer, make_engine, model, moe, reference, seq   # noqa: E402

TOL = 1e-4


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        sd = oracle.random_model(cfg, seed=len(name))
        d = tmp_path_factory.mktemp("m") / name
        oracle.write_model(cfg, sd, d)
        out[name] = (cfg, sd, d)
    return out


@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt_and_decode(folders, name):
    cfg, sd, d = folders[name]
    toks = {"a": seq(70, cfg["vocab"], 1)}
    want = reference(cfg, sd, toks)
    assert err(feed(make_engine(d), toks, [[("a", 70)]])["a"], want["a"]) < TOL
    assert err(feed(make_engine(d), toks, [[("a", 1)]] * 70)["a"], want["a"]) < TOL


@pytest.mark.parametrize("sizes", [(2,), (3, 1, 2), (16,), (17, 15), (5, 33, 2)])
def test_portions(folders, sizes):
    cfg, sd, d = folders["odd"]
    toks = {"a": seq(67, cfg["vocab"], 2)}
    got = feed(make_engine(d), toks, [[("a", n)] for n in cut(67, sizes)])
    assert err(got["a"], reference(cfg, sd, toks)["a"]) < TOL


def test_batches_of_unequal_requests_and_reuse(folders):
    """Portions beside single tokens; requests that pause; pages and slots that were used by finished requests."""
    cfg, sd, d = folders["even"]
    toks = {"a": seq(60, cfg["vocab"], 3), "b": seq(21, cfg["vocab"], 4), "c": seq(1, cfg["vocab"], 5), "d": seq(50, cfg["vocab"], 6),
            "e": seq(37, cfg["vocab"], 7), "f": seq(18, cfg["vocab"], 8)}
    steps = [[("a", 29), ("b", 2), ("c", 1)], [("b", 1), ("a", 2), ("d", 17)], [("d", 1), ("b", 1)], [("a", 1), ("d", 16), ("b", 17)],   # b, c end
             [("e", 3), ("a", 27), ("d", 1)], [("e", 33), ("f", 1), ("a", 1), ("d", 14)], [("d", 1), ("f", 16), ("e", 1)], [("f", 1)]]    # a, e, d end
    eng = make_engine(d, tokens=192)
    free, want = None, reference(cfg, sd, toks)
    for _ in range(2):
        got = feed(eng, toks, steps)
        for k in toks:
            assert err(got[k], want[k]) < TOL, k
        now = (eng.alloc.available(), len(eng.state.free), len(eng.free_slots))
        assert free in (None, now)                  # everything was given back
        free = now
    assert not eng.running


# ---------------------------------------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("mixer", [A_EVEN, A_ODD, attn(2, 1, 12, 30, 16, 4), attn(3, 3, 8, 3, 500, 0), attn(4, 2, 6, 6, 17, 6, scaling=(32.0, 2.0, 3.0, 40))])
def test_attention_alone(tmp_path, mixer):
    cfg = model(40, 50, layer(mixer), taps=1)
    sd = oracle.random_model(cfg, 5)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(80, 50, 9), "b": seq(33, 50, 10)}
    got = feed(make_engine(tmp_path / "m"), toks, [[("a", 50), ("b", 16)], [("a", 1), ("b", 15)], [("a", 28), ("b", 1)], [("b", 1), ("a", 1)]])
    want = reference(cfg, sd, toks)
    assert max(err(got[k], want[k]) for k in toks) < TOL


def test_frequency_scaling_has_three_ranges():
    from polyrl_b200.ops import mixers as M

    rot = dict(base=5000.0, dims=24, scaling=dict(factor=7.0, low=1.5, high=5.0, original=300))
    got = M.scaled_frequencies(24, 5000.0, rot["scaling"], "cpu")
    assert torch.allclose(got, torch.tensor(oracle.frequencies(rot), dtype=oracle.D), rtol=1e-12)
    plain = M.rope_frequencies(24, 5000.0, "cpu")
    r = plain / got
    assert (r == 1).any() and torch.isclose(r, torch.tensor(7.0, dtype=oracle.D)).any() and ((r > 1.01) & (r < 6.9)).any()
    assert torch.equal(M.scaled_frequencies(24, 5000.0, None, "cpu"), plain)


def far_model(window):
    """One attention layer in which token 1 asks, token 2 is the key that answers in the first map and token 3 the one of the second (their scores
    stand out by e^8) and every other pair scores zero."""
    d = 8
    cfg = model(16, 12, layer(attn(1, 1, d, 8, window, 2, 100.0, 1.0)), taps=1)
    sd = oracle.random_model(cfg, 11)
    e = torch.full((12, 16), -1.0 / 3, dtype=oracle.D)             # rows whose layer norm keeps one entry standing out
    for t in range(12):
        e[t, t] = 5.0
    sd["embed"], sd["l0.norm1"], sd["l0.canon1"] = e, torch.ones(16, dtype=oracle.D), torch.zeros(16, 1, dtype=oracle.D)
    sd["l0.dwa"] = torch.tensor([0.0, 1.0], dtype=oracle.D)
    q, k = torch.zeros(2 * d, 16, dtype=oracle.D), torch.zeros(2 * d, 16, dtype=oracle.D)
    for m in range(2):                                             # the rotation turns entries 0 and 1 of a map only
        q[m * d + 2, 1] = q[m * d + 3, 5] = 4.0
        k[m * d + 2, 2 + m] = 4.0
        for t in [x for x in range(12) if x != 2 + m]:
            k[m * d + 4 + t % 4, t] = 4.0
    sd["l0.mix.q"], sd["l0.mix.k"] = q, k
    for n in ("q.b", "k.b", "v.b"):
        sd[f"l0.mix.{n}"] = torch.zeros_like(sd[f"l0.mix.{n}"])
    for n in ("q.norm", "k.norm"):
        sd[f"l0.mix.{n}"] = torch.ones(d, dtype=oracle.D)
    return cfg, sd


@pytest.mark.parametrize("window", [1, 2, 16, 17, 33, 40])
def test_keys_just_inside_and_outside_the_window(tmp_path, window):
    cfg, sd = far_model(window)
    oracle.write_model(cfg, sd, tmp_path / "m")
    sd = {k: t.to(torch.bfloat16).to(oracle.D) for k, t in sd.items()}
    for at in (0, 1, 15, 16, 31, 32):
        for key in (2, 3):
            t = [4 + x for x in seq(100, 8, at)]
            t[at] = key
            asks = sorted({min(99, at + max(window - 1, 1)), min(99, at + window), min(99, at + window + 1), 98, 99})      # just inside, just outside, far
            for q in asks:
                t[q] = 1
            want = reference(cfg, sd, {"a": t})["a"]
            hidden = list(t)
            hidden[at] = 4                                         # the same sequence without that key
            diff = (reference(cfg, sd, {"a": hidden})["a"] - want).pow(2).mean(-1).sqrt()
            for q in asks:
                assert (diff[q] > 0.02) == oracle.visible(q, at, window), (at, q, diff[q])
            for steps in ([100], cut(100, (33, 16, 1)), cut(100, (2,)), [at + 1] + [1] * (99 - at)):
                got = feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in steps])["a"]
                assert err(got, want) < TOL, (at, steps)


def test_second_map_counts_with_its_weight(folders):
    """lambda far from the constant, other maps, other sign."""
    cfg, sd, d = folders["even"]
    toks = {"a": seq(30, cfg["vocab"], 1)}
    base = reference(cfg, sd, toks)["a"]
    for n, f in (("lq1", 3.0), ("lk2", -2.0), ("lq2", 0.0)):
        other = dict(sd)
        other[f"l0.mix.{n}"] = other[f"l0.mix.{n}"] * f + 0.3
        assert err(reference(cfg, other, toks)["a"], base) > 1e-2, n
    other = {k: (t * 4 if k.split(".")[-1] in ("lq1", "lk1") else t).to(torch.bfloat16).to(oracle.D) for k, t in sd.items()}
    folder = d.parent / "lam"
    oracle.write_model(cfg, other, folder)
    assert err(feed(make_engine(folder), toks, [[("a", 30)]])["a"], reference(cfg, other, toks)["a"]) < TOL


def test_input_convolutions_across_cuts(tmp_path):
    """Strong taps; both sublayers read their own; a token at a portion's edge is seen by the next portion's first tokens."""
    cfg = model(24, 30, layer(attn(2, 1, 6, 6, 1, 2), dense(20)), layer(attn(2, 1, 6, 6, 1, 2), dense(20)), taps=4)
    sd = oracle.random_model(cfg, 3)
    for k in sd:
        if "canon" in k:
            sd[k] = (3 * sd[k]).to(torch.bfloat16).to(oracle.D)
    oracle.write_model(cfg, sd, tmp_path / "m")
    t = seq(60, 30, 12)
    want = reference(cfg, sd, {"a": t})["a"]
    other = list(t)
    other[20] = (t[20] + 7) % 30
    moved = (reference(cfg, sd, {"a": other})["a"] - want).abs().amax(-1) > 1e-6
    assert moved.nonzero().flatten().tolist() == list(range(20, 27))         # three earlier inputs in each of two layers
    for k in ("l0.canon1", "l0.canon2", "l1.canon1"):
        assert err(reference(cfg, dict(sd, **{k: torch.zeros_like(sd[k])}), {"a": t})["a"], want) > 1e-2
    for sizes in ((60,), (2,), (3, 1), (21, 1, 38), (1,), (4,)):
        assert err(feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in cut(60, sizes)])["a"], want) < TOL, sizes


def test_depth_average_reads_every_earlier_result(folders):
    cfg, sd, d = folders["odd"]
    toks = {"a": seq(20, cfg["vocab"], 1)}
    base = reference(cfg, sd, toks)["a"]
    for i in range(len(cfg["layers"])):
        for j in range(i + 2):
            other = dict(sd)
            other[f"l{i}.dwa"] = other[f"l{i}.dwa"].clone()
            other[f"l{i}.dwa"][j] += 0.5
            assert err(reference(cfg, other, toks)["a"], base) > 1e-2, (i, j)


@pytest.mark.parametrize("act", [(1.0, 0.0, 0.0, 0.0), (0.0, 1.0, 0.0, 0.0), (0.0, 0.0, 1.0, 0.0), (0.2, -0.3, 0.4, 0.7)])
def test_polynomial_activation(act):
    from polyrl_b200.ops import mixers as M

    z = torch.randn(5, 37, dtype=torch.float32) * 2
    want = oracle.poly_norm(z.double(), act, 1e-3)
    assert (M.poly_norm(z, torch.tensor(act), 1e-3) - want).abs().max() < 1e-5


@pytest.mark.parametrize("n,top,ff,shared", [(5, 2, 24, None), (4, 4, 128, 16), (9, 1, 7, 130), (1, 1, 8, 8)])
def test_experts_alone(tmp_path, n, top, ff, shared):
    """Weights on the experts' inputs, not renormalised: experts are not linear, so a weight on the output would show."""
    cfg = model(32, 40, layer(attn(1, 1, 2, 2, 1, 2), moe(n, top, ff, shared)), taps=1)
    sd = oracle.random_model(cfg, n)
    for k in sd:
        if ".mlp." in k:
            sd[k] = ((0.25 if k.endswith("router") else 2) * sd[k]).to(torch.bfloat16).to(oracle.D)      # scores well below one
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(40, 40, 1)}
    want = reference(cfg, sd, toks)["a"]
    assert err(feed(make_engine(tmp_path / "m"), toks, [[("a", 25)], [("a", 1)], [("a", 14)]])["a"], want) < TOL
    h, mlp = torch.randn(6, 32, dtype=oracle.D), {k[len("l0.mlp."):]: t for k, t in sd.items() if ".mlp." in k}
    pick, s = oracle.route(h, mlp["router"], top)
    outside = torch.stack([sum(g * oracle.gated(h[t], mlp, f"e{e}.") for e, g in zip(pick[t].tolist(), s[t])) for t in range(6)])
    inside = oracle.mixture(h, {k: v for k, v in mlp.items() if "shared" not in k}, dict(router=dict(top=top)))
    assert (outside - inside).norm() > 0.02 * inside.norm()


# ---------------------------------------------------------------------------------------------- the framework around it
def greedy_oracle(cfg, sd, prompt, n):
    t = list(prompt)
    for _ in range(n):
        t.append(int(oracle.forward(cfg, sd, t)[-1].argmax()))
    return t[len(prompt):]


@pytest.mark.parametrize("chunk", [16384, 7])
@pytest.mark.parametrize("native", ["1", "0"])
def test_greedy_generation_through_the_scheduler(folders, chunk, native, monkeypatch):
    monkeypatch.setenv("POLYRL_NATIVE_SCHED", native)
    monkeypatch.setenv("POLYRL_NATIVE_KV", native)
    cfg, sd, d = folders["odd"]
    prompts = [seq(n, cfg["vocab"], n) for n in (1, 5, 16, 23, 9)]
    want = [greedy_oracle(cfg, sd, p, 12) for p in prompts]
    eng = make_engine(d, seqs=3, max_len=64, max_prefill_tokens=chunk)           # five requests through three slots
    for _ in range(2):
        out = eng.generate(prompts, dict(max_new_tokens=12, temperature=0.0))
        assert [g[0].output_ids for g in out] == want
    assert len(eng.state.free) == 3 and not eng.running


def test_offline_generation_entry_point(folders):
    from polyrl_b200.trainer.main_generation import generate

    cfg, sd, d = folders["even"]
    rows = [{"prompt": seq(n, cfg["vocab"], n)} for n in (4, 19)]
    out = generate(str(d), rows, temperature=0.0, response_length=6, prompt_length=32, device="cpu")
    assert [r["response_ids"][0] for r in out] == [greedy_oracle(cfg, sd, r["prompt"], 6) for r in rows]


def test_sample_groups_share_the_prompt(folders):
    cfg, sd, d = folders["even"]
    prompt = seq(21, cfg["vocab"], 2)
    want = greedy_oracle(cfg, sd, prompt, 10)
    out = make_engine(d, seqs=4, max_len=64).generate([prompt], dict(max_new_tokens=10, temperature=0.0, n=3))
    assert [r.output_ids for r in out[0]] == [want] * 3


def test_config_registry_loader_and_export_round_trip(folders, tmp_path):
    from polyrl_b200.models import ModelConfig, get_model_config
    from polyrl_b200.models.hf_io import load_state_dict, save_hf

    for name in CONFIGS:
        cfg, sd, d = folders[name]
        mc = get_model_config(str(d))
        assert (mc.family, mc.num_layers, mc.vocab_size, mc.hidden_size) == ("hybrid", len(cfg["layers"]), cfg["vocab"], cfg["width"])
        assert mc.input_conv == cfg["canon"]["taps"] and mc.num_params() == sum(t.numel() for t in sd.values())
        assert ModelConfig(**json.loads(json.dumps(mc.to_dict()))) == mc
        save_hf(load_state_dict(mc, d), mc, tmp_path / name)
        back = oracle.read_safetensors(tmp_path / name / "model.safetensors")
        assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
        assert get_model_config(str(tmp_path / name)) == mc
    cfg = folders["even"][0]
    first, second = cfg["layers"][:2]
    for bad in ([dict(first, type="conv")], [first, dict(second, weights_of=0)], [dict(first, mlp=dict(kind="sparse", ff=8))],
                [dict(first, mixer=dict(first["mixer"], kv_heads=3))], [dict(second, mlp=moe(3, 4, 8))], [dict(first, mixer=dict(first["mixer"], mask=dict(size=0)))]):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(dict(cfg, layers=bad))


def test_caches_are_sized(folders):
    from polyrl_b200.models import get_model_config, hybrid

    for name in ("odd", "even"):
        cfg, sd, d = folders[name]
        mc = get_model_config(str(d))
        eng = make_engine(d, dtype=torch.bfloat16)
        eng.init_kv_cache()
        tok, slot = hybrid.cache_bytes(mc, torch.bfloat16)
        pools = [t for c in eng.k_cache for k, t in c.items() if k.endswith("pool")]
        states = [t for c in eng.k_cache for k, t in c.items() if not k.endswith("pool")]
        assert sum(t[0].numel() * 2 for t in pools) == 16 * tok and sum(t[0].numel() * t.element_size() for t in states) == slot
        toks = {"a": seq(40, cfg["vocab"], 2)}
        got = feed(eng, toks, [[("a", 21)], [("a", 1)], [("a", 18)]])["a"]
        d_ = (got - reference(cfg, sd, toks)["a"]).pow(2).mean(-1).sqrt()
        assert d_.median() < 0.05


def test_trace_replay(folders, tmp_path):
    from polyrl_b200.rollout import trace

    cfg, sd, d = folders["even"]
    t = seq(20, cfg["vocab"], 3)
    want = oracle.forward(cfg, sd, t)
    lines = [dict(step=0, entries=[dict(id="a", tokens=t[:7], want=[6, 2])], end=[]), dict(step=1, entries=[dict(id="a", tokens=t[7:8], want=[])], end=[]),
             dict(step=5, entries=[dict(id="a", tokens=t[8:], want=[11]), dict(id="b", tokens=t[:1], want=[0])], end=["a", "b"])]
    eng = trace.load_engine(str(d), "float32", 64, "cpu")
    said = []
    trace.replay(eng, io.StringIO("\n".join(json.dumps(x) for x in lines)), tmp_path, emit=said.append)
    assert said == ["done 0", "done 1", "done 5"]

    def rows(n):
        return torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, cfg["vocab"]).double()

    assert err(rows(0), want[[6, 2]]) < TOL and err(rows(5), want[[19, 0]]) < TOL


def test_parallel_blocks_with_other_parts():
    """The block's options are independent of the design: RMS norm, no convolution, no scales, no averages, other mixers and feed-forwards."""
    from polyrl_b200.models import ModelConfig, TransformerWeights
    from polyrl_b200.rollout.engine import RolloutEngine

    delta = dict(kind="delta", sizes=dict(heads=2, kv_heads=1, dim=6, vdim=5, conv=3), ff=24, act="gelu")
    base = dict(family="hybrid", vocab_size=40, hidden_size=24, intermediate_size=24, num_layers=2, num_heads=1, num_kv_heads=1, hf_model_type="", eos_token_id=-1,
                layers=(dict(delta, weights_of=0), dict(delta, ff=0, weights_of=1)))
    toks = {"a": seq(30, 40, 1)}
    for kw in ({}, dict(layer_norm=True), dict(input_conv=3), dict(layer_scale=True), dict(depth_average=True)):
        cfg = ModelConfig(**base, parallel_block=True, **kw)
        w = TransformerWeights(cfg, seed=1)
        outs = []
        for sizes in ((30,), (7, 1, 2)):
            eng = RolloutEngine(cfg, "cpu", max_num_seqs=2, max_model_len=64)
            eng.set_weights(w.embed, w.layers, w.head)
            outs.append(feed(eng, toks, [[("a", n)] for n in cut(30, sizes)])["a"])
        assert torch.isfinite(outs[0]).all() and err(outs[1], outs[0]) < TOL
    with pytest.raises(ValueError):
        ModelConfig(**base, input_conv=3)


def test_presets():
    from polyrl_b200.models import TransformerWeights, get_model_config
    from polyrl_b200.rollout.engine import RolloutEngine

    cfg = get_model_config("tiny-mabedra")
    w = TransformerWeights(cfg, seed=1)
    assert cfg.num_params() == sum(t.numel() for _, t in w.named_tensors())
    assert w.layers[1]["depth"].tolist() == [0.0, 0.0, 1.0] and (w.layers[1]["ls2"] == 1).all() and (w.layers[0]["map_mix"] == 0).all()
    eng = RolloutEngine(cfg, "cpu", max_num_seqs=2, max_model_len=32)
    eng.set_weights(w.embed, w.layers, w.head)
    assert len(eng.generate([[3, 4, 5]], dict(max_new_tokens=4, temperature=1.0))[0][0].output_ids) == 4
    assert get_model_config("mabedra-7b").num_params() > 6e9 and math.isclose(float(eng.layer_w[0]["lam"]), cfg.layers[0]["sizes"]["diff"], rel_tol=1e-6)
