"""Lanilix stacks through the framework's configuration, loader, scheduler, cache / state manager and step functions, on CPU in fp32,
against the plain oracle (tests/lanilix_oracle.py)."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(__file__))
import lanilix_oracle as oracle                       # noqa: E402
from lanilix_util import ATTN_EVEN, ATTN_ODD, CONFIGS, DELTA_EVEN, DELTA_ODD, attn, cut, err, feed, layer, make_engine, model, reference, seq   # noqa: E402

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
@pytest.mark.parametrize("kind,mixer", [("delta", DELTA_EVEN), ("delta", DELTA_ODD), ("attention", ATTN_EVEN), ("attention", ATTN_ODD),
                                        ("attention", attn(2, 1, 12, 16, 16, 4)), ("attention", attn(3, 3, 8, 500, 0, 0))])
def test_single_layer(tmp_path, kind, mixer):
    cfg = model(40, 50, layer(kind, mixer))
    sd = oracle.random_model(cfg, 5)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(80, 50, 9), "b": seq(33, 50, 10)}
    got = feed(make_engine(tmp_path / "m"), toks, [[("a", 50), ("b", 16)], [("a", 1), ("b", 15)], [("a", 28), ("b", 1)], [("b", 1), ("a", 1)]])
    want = reference(cfg, sd, toks)
    assert max(err(got[k], want[k]) for k in toks) < TOL


def test_oracle_recurrence_matches_its_closed_form():
    """One key, no decay, full writes: the state answers the key with the last value."""
    k = oracle.unit(torch.randn(1, 1, 5, dtype=oracle.D)).expand(6, 1, 5)
    v = torch.randn(6, 1, 4, dtype=oracle.D)
    one = torch.ones(6, 1, dtype=oracle.D)
    o, _ = oracle.delta_scan(k, k, v, one, one)
    assert (o - v).abs().max() < 1e-5


def far_model(window, keep):
    """One attention layer in which token 1 asks, token 2 is the key that answers (its score stands out by e^8) and every other pair scores zero."""
    cfg = model(16, 12, layer("attention", attn(1, 1, 8, window, keep, 2, 100.0, 1.0)))
    sd = oracle.random_model(cfg, 11)
    e = torch.zeros(12, 16, dtype=oracle.D)
    for t in range(12):
        e[t, t] = 2.0
    sd["embed"] = e
    q, k = torch.zeros(8, 16, dtype=oracle.D), torch.zeros(8, 16, dtype=oracle.D)
    q[2, 1] = 1.0                                                  # the rotation turns entries 0 and 1 only
    q[3, [0] + list(range(2, 12))] = 1.0
    k[2, 2] = 1.0
    for t in [0, 1] + list(range(3, 12)):
        k[4 + t % 4, t] = 1.0
    sd["l0.mix.q"], sd["l0.mix.k"] = q, k
    for n in ("q.norm", "k.norm"):
        sd[f"l0.mix.{n}"] = torch.ones(8, dtype=oracle.D)
    return cfg, sd


@pytest.mark.parametrize("window,keep", [(16, 0), (17, 3), (33, 16), (40, 1), (1, 2)])
def test_far_keys_at_window_page_and_kept_edges(tmp_path, window, keep):
    cfg, sd = far_model(window, keep)
    oracle.write_model(cfg, sd, tmp_path / "m")
    for at in {0, 1, max(keep - 1, 0), keep, keep + 1, 15, 16, 31, 32}:
        t = [3 + x for x in seq(100, 9, at)]
        t[at] = 2
        asks = sorted({min(99, at + max(window - 1, 1)), min(99, at + window), min(99, at + window + 1), 98, 99})      # just inside, just outside, far
        for q in asks:
            t[q] = 1
        want = reference(cfg, sd, {"a": t})["a"]
        hidden = list(t)
        hidden[at] = 3                                             # the same sequence without that key
        diff = (reference(cfg, sd, {"a": hidden})["a"] - want).pow(2).mean(-1).sqrt()
        for q in asks:
            assert (diff[q] > 0.05) == oracle.visible(q, at, window, keep), (at, q)
        for steps in ([100], cut(100, (33, 16, 1)), cut(100, (2,)), [at + 1] + [1] * (99 - at)):
            got = feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in steps])["a"]
            assert err(got, want) < TOL, (at, steps)


def test_kept_tokens_keep_their_positions(tmp_path):
    """Rotation over the whole width: a kept key is turned by its true position however far the query is."""
    cfg = model(24, 30, layer("attention", attn(2, 1, 8, 5, 3, 8, 30.0, 1.5)))
    sd = oracle.random_model(cfg, 2)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(120, 30, 4)}
    want = reference(cfg, sd, toks)["a"]
    for sizes in ((120,), (50, 1), (2, 9)):
        assert err(feed(make_engine(tmp_path / "m"), toks, [[("a", n)] for n in cut(120, sizes)])["a"], want) < TOL


def test_the_recurrence_remembers_far_tokens_and_portion_edges(tmp_path):
    """Slow decays, so that a token at a portion's or page's edge is still read much later; convolution taps across the cut."""
    cfg = model(24, 30, layer("delta", dict(heads=2, kv_heads=1, dim=12, vdim=6, conv=4)))
    sd = oracle.random_model(cfg, 3)
    sd["l0.mix.A_log"] = torch.full((2,), -7.0, dtype=oracle.D)
    sd["l0.mix.b"] *= 0.25
    oracle.write_model(cfg, sd, tmp_path / "m")
    t = seq(130, 30, 12)
    want = reference(cfg, sd, {"a": t})["a"]
    for at in (0, 2, 3, 15, 16, 63, 64):
        other = list(t)
        other[at] = (t[at] + 7) % 30
        assert err(reference(cfg, sd, {"a": other})["a"][129:], want[129:]) > 1e-4
    for sizes in ((130,), (2,), (3, 1), (64, 1, 63), (1,)):
        got = feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in cut(130, sizes)])["a"]
        assert err(got, want) < 2e-5, sizes


def test_feed_forward_clamps_and_offsets(tmp_path):
    """Pre-activations on both sides of both limits; norm weights far from zero."""
    cfg = model(16, 20, layer("delta", DELTA_ODD, 24, 0.3), layer("delta", DELTA_ODD, 128, 2.0), eps=0.1)
    sd = oracle.random_model(cfg, 8)
    for k in sd:
        if k.endswith(("mlp.gate", "mlp.up")):
            sd[k] = (3 * sd[k]).to(torch.bfloat16).to(oracle.D)
        if "norm1" in k or "norm2" in k or k == "final.norm":
            sd[k] = (sd[k] - 0.6).to(torch.bfloat16).to(oracle.D)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(30, 20, 1)}
    want = reference(cfg, sd, toks)["a"]
    for i, lim in ((0, 1e9), (1, 1e9)):                            # both limits bite
        other = json.loads(json.dumps(cfg))
        other["layers"][i]["mlp"]["limit"] = lim
        assert err(reference(other, sd, toks)["a"], want) > 1e-2
    assert err(feed(make_engine(tmp_path / "m"), toks, [[("a", 9)], [("a", 21)]])["a"], want) < TOL


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

    for name in ("odd", "even"):
        cfg, sd, d = folders[name]
        mc = get_model_config(str(d))
        assert (mc.family, mc.num_layers, mc.vocab_size, mc.hidden_size) == ("hybrid", len(cfg["layers"]), cfg["vocab"], cfg["width"])
        assert mc.num_params() == sum(t.numel() for t in sd.values())
        assert ModelConfig(**json.loads(json.dumps(mc.to_dict()))) == mc
        save_hf(load_state_dict(mc, d), mc, tmp_path / name)
        back = oracle.read_safetensors(tmp_path / name / "model.safetensors")
        assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
        assert get_model_config(str(tmp_path / name)) == mc
    first, second = cfg["layers"][:2]
    for bad in ([dict(first, type="conv")], [first, dict(second, weights_of=0)], [dict(first, mixer=dict(first["mixer"], vdim=first["mixer"]["vdim"] + 2))],
                [dict(first, mlp=dict(kind="sparse", ff=8, limit=1.0))], [dict(first, mixer=dict(first["mixer"], kv_heads=3))]):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(dict(cfg, layers=bad))


def test_layers_that_reuse_weights_keep_their_own_state(folders):
    cfg, sd, d = folders["odd"]
    eng = make_engine(d)
    eng.init_kv_cache()
    assert eng.layer_w[3] is eng.layer_w[1] and eng.layer_w[4] is eng.layer_w[0]
    assert eng.k_cache[3]["k_pool"].data_ptr() != eng.k_cache[1]["k_pool"].data_ptr()
    assert eng.k_cache[4]["S"].data_ptr() != eng.k_cache[0]["S"].data_ptr()


def test_bf16_caches_are_padded_and_sized(folders):
    from polyrl_b200.models import get_model_config, hybrid

    cfg, sd, d = folders["odd"]
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


def test_presets():
    from polyrl_b200.models import TransformerWeights, get_model_config
    from polyrl_b200.rollout.engine import RolloutEngine

    cfg = get_model_config("tiny-lanilix")
    w = TransformerWeights(cfg, seed=1)
    assert w.layers[3] is w.layers[0] and cfg.num_params() == sum(t.numel() for _, t in w.named_tensors())
    assert (w.layers[1]["pre1"] == 0).all() and (w.layers[1]["q_norm"] == 1).all() and (w.head["norm_w"] == 0).all()
    eng = RolloutEngine(cfg, "cpu", max_num_seqs=2, max_model_len=32)
    eng.set_weights(w.embed, w.layers, w.head)
    assert len(eng.generate([[3, 4, 5]], dict(max_new_tokens=4, temperature=1.0))[0][0].output_ids) == 4
    assert get_model_config("lanilix-4b").num_params() > 3e9
