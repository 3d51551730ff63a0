"""Ludesun stacks through the framework's configuration, loader, scheduler, cache / state manager and step functions, on CPU in fp32,
against the plain oracle (tests/ludesun_oracle.py)."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(__file__))
import ludesun_oracle as oracle                       # noqa: E402
from ludesun_util import CONFIGS, EVEN, LATENT_EVEN, MAMBA_EVEN, MLSTM_EVEN, ODD, cut, err, feed, layer, make_engine, model, reference, seq   # noqa: E402

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
    whole = feed(make_engine(d), toks, [[("a", 70)]])
    assert err(whole["a"], want["a"]) < TOL
    one_by_one = feed(make_engine(d), toks, [[("a", 1)]] * 70)
    assert err(one_by_one["a"], want["a"]) < TOL


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
    free = None
    for _ in range(2):
        got = feed(eng, toks, steps)
        want = reference(cfg, sd, toks)
        for k in toks:
            assert err(got[k], want[k]) < TOL, k
        now = (eng.alloc.available(), len(eng.state.free), len(eng.free_slots))
        assert free in (None, now)                  # everything was given back
        free = now
    assert not eng.running


def test_pool_exhaustion_is_an_error(folders):
    cfg, _, d = folders["odd"]
    eng = make_engine(d, seqs=2, max_len=64, tokens=48)
    a, b, c = (eng.open(x) for x in "abc")
    eng.extend([(a, seq(32, cfg["vocab"], 1), []), (b, [1], [])])
    with pytest.raises((MemoryError, RuntimeError)):
        eng.extend([(c, [1], [])])                  # no third slot
    with pytest.raises((MemoryError, RuntimeError)):
        eng.extend([(a, [1] * 16, [])])             # no page left
    eng.close(b)
    assert eng.extend([(a, [1] * 16, [15])]).shape == (1, cfg["vocab"])
    with pytest.raises(ValueError):
        eng.extend([(a, [1] * 32, [])])             # longer than max_model_len


# ---------------------------------------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("kind,mixer", [("mamba2", MAMBA_EVEN), ("latent_attention", LATENT_EVEN), ("mlstm", MLSTM_EVEN)])
def test_single_layer(tmp_path, kind, mixer):
    cfg = model(40, 50, layer(kind, mixer))
    sd = oracle.random_model(cfg, 5)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(80, 50, 9), "b": seq(33, 50, 10)}
    got = feed(make_engine(tmp_path / "m"), toks, [[("a", 50), ("b", 16)], [("a", 1), ("b", 15)], [("a", 28), ("b", 1)], [("b", 1), ("a", 1)]])
    want = reference(cfg, sd, toks)
    assert max(err(got[k], want[k]) for k in toks) < TOL


def far_model(sink):
    """One latent layer whose score of the pair (token 1 queries, token 2 is the key) stands out; everything else scores near zero."""
    m = dict(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8, q_rank=8, scale=6.0, rot=dict(base=100.0, dims=2))
    cfg = model(16, 12, layer("latent_attention", m))
    sd = oracle.random_model(cfg, 11)
    e = torch.zeros(12, 16, dtype=oracle.D)
    e[1, 0], e[2, 1] = 2.0, 2.0
    for t in [0] + list(range(3, 12)):
        e[t, 2 + t % 8] = 2.0
    sd["embed"] = e
    for k in ("dq", "dkv", "uq", "uk", "uv"):
        sd[f"l0.mix.{k}"] = torch.zeros_like(sd[f"l0.mix.{k}"])
    sd["l0.mix.dq"][:, 0] = 1.0                                    # only token 1 asks
    sd["l0.mix.dkv"][0, 1] = 1.0                                   # token 2's latent is e_0, the others' live in 1..7
    for i in range(1, 8):
        sd["l0.mix.dkv"][i, 2 + i] = 1.0
    sd["l0.mix.uq"][0, :] = 0.25
    sd["l0.mix.uk"][0, 0] = 1.0
    sd["l0.mix.uv"] = torch.eye(8, dtype=oracle.D)
    sd["l0.mix.sink"] = torch.full((1,), sink, dtype=oracle.D)
    return cfg, sd


@pytest.mark.parametrize("sink", [-3.0, 4.0])
def test_far_keys_and_page_borders(tmp_path, sink):
    cfg, sd = far_model(sink)
    oracle.write_model(cfg, sd, tmp_path / "m")
    for at in (0, 1, 14, 15, 16, 17, 31, 32, 47, 63):              # place of the key that matters
        t = seq(100, 9, at)
        t = [x + 3 for x in t]
        t[at] = 2
        for q in (at + 1, 64, 80, 99):
            t[q] = 1
        toks = {"a": t}
        want = reference(cfg, sd, toks)["a"]
        hidden = list(t)
        hidden[at] = 3                                             # the same sequence without that key
        assert err(reference(cfg, sd, {"a": hidden})["a"][99:], want[99:]) > 0.05
        for steps in ([100], cut(100, (33, 16, 1)), [60] + [1] * 40):
            got = feed(make_engine(tmp_path / "m"), toks, [[("a", n)] for n in steps])["a"]
            assert err(got, want) < TOL, (at, steps)


def test_recurrences_remember_far_tokens_and_portion_edges(tmp_path):
    """Slow decays, so that a token at a portion's or page's edge is still read much later; convolution taps across the cut."""
    cfg = model(24, 30, layer("mamba2", dict(heads=2, vdim=6, state=4, groups=2, conv=4, norm_groups=2)),
                layer("mlstm", dict(heads=2, dim=5, vdim=4, gate_cap=9.0)))
    sd = oracle.random_model(cfg, 3)
    sd["l0.mix.A_log"] = torch.full((2,), -6.0, dtype=oracle.D)
    sd["l1.mix.f.b"] = torch.full((2,), 8.0, dtype=oracle.D)
    sd["l1.mix.f"] = torch.zeros_like(sd["l1.mix.f"])
    oracle.write_model(cfg, sd, tmp_path / "m")
    t = seq(150, 30, 12)
    want = reference(cfg, sd, {"a": t})["a"]
    for at in (0, 2, 3, 15, 16, 63, 64):
        other = list(t)
        other[at] = (t[at] + 7) % 30
        assert err(reference(cfg, sd, {"a": other})["a"][149:], want[149:]) > 1e-3
    for sizes in ((150,), (2,), (3, 1), (64, 1, 63), (1,)):
        got = feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in cut(150, sizes)])["a"]
        assert err(got, want) < TOL, sizes


def test_mlstm_running_maximum_starts_at_zero(tmp_path):
    """Input gates far below zero: with m starting at 0 the state stays tiny against the floor exp(-m)."""
    cfg = model(16, 20, layer("mlstm", dict(heads=2, dim=4, vdim=4, gate_cap=20.0)))
    sd = oracle.random_model(cfg, 4)
    sd["l0.mix.i.b"] = torch.tensor([-9.0, 5.0], dtype=oracle.D)
    sd["l0.mix.f.b"] = torch.tensor([-4.0, 1.0], dtype=oracle.D)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(40, 20, 1)}
    want = reference(cfg, sd, toks)["a"]
    for sizes in ((40,), (7, 2), (1,)):
        assert err(feed(make_engine(tmp_path / "m"), toks, [[("a", n)] for n in cut(40, sizes)])["a"], want) < TOL


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


def test_release_and_resume(folders):
    cfg, sd, d = folders["even"]
    eng = make_engine(d, max_len=64)
    a = eng.generate([[1, 2, 3]], dict(max_new_tokens=6, temperature=0.0))[0][0].output_ids
    eng.release_memory()
    assert eng.state is None
    eng.resume_memory()
    assert eng.generate([[1, 2, 3]], dict(max_new_tokens=6, temperature=0.0))[0][0].output_ids == a


def test_config_registry_loader_and_export_round_trip(folders, tmp_path):
    from polyrl_b200.models import ModelConfig, get_model_config
    from polyrl_b200.models.hf_io import load_state_dict, save_hf

    cfg, sd, d = folders["odd"]
    mc = get_model_config(str(d))
    assert (mc.family, mc.num_layers, mc.vocab_size, mc.hidden_size) == ("hybrid", 5, cfg["vocab"], cfg["width"])
    assert mc.num_params() == sum(t.numel() for t in sd.values())
    assert ModelConfig(**json.loads(json.dumps(mc.to_dict()))) == mc
    ours = load_state_dict(mc, d)
    save_hf(ours, mc, tmp_path / "x")
    back = oracle.read_safetensors(tmp_path / "x" / "model.safetensors")
    assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) for k in sd)
    assert get_model_config(str(tmp_path / "x")) == mc
    bad = dict(cfg, layers=[dict(cfg["layers"][0], type="conv")])
    with pytest.raises(ValueError):
        ModelConfig.from_hf_config(bad)
    with pytest.raises(ValueError):
        ModelConfig.from_hf_config(dict(cfg, layers=[cfg["layers"][0], dict(cfg["layers"][1], weights_of=0)]))


def test_layers_that_reuse_weights_keep_their_own_state(folders):
    cfg, sd, d = folders["odd"]
    eng = make_engine(d)
    eng.init_kv_cache()
    assert eng.layer_w[3] is eng.layer_w[1] and eng.layer_w[4] is eng.layer_w[0]
    assert eng.k_cache[3]["pool"].data_ptr() != eng.k_cache[1]["pool"].data_ptr()
    assert eng.k_cache[4]["S"].data_ptr() != eng.k_cache[0]["S"].data_ptr()


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
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "5.f32"]

    def rows(n):
        return torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).reshape(-1, cfg["vocab"]).double()

    assert err(rows(0), want[[6, 2]]) < TOL and err(rows(5), want[[19, 0]]) < TOL


def test_presets_and_unsupported_paths():
    from polyrl_b200.models import TransformerWeights, get_model_config, layer_forward
    from polyrl_b200.rollout.engine import RolloutEngine

    cfg = get_model_config("tiny-ludesun")
    w = TransformerWeights(cfg, seed=1)
    assert w.layers[3] is w.layers[0] and cfg.num_params() == sum(t.numel() for _, t in w.named_tensors())
    eng = RolloutEngine(cfg, "cpu", max_num_seqs=2, max_model_len=32)
    eng.set_weights(w.embed, w.layers, w.head)
    r = eng.generate([[3, 4, 5]], dict(max_new_tokens=4, temperature=1.0))[0][0]
    assert len(r.output_ids) == 4
    with pytest.raises(NotImplementedError):
        layer_forward(cfg, w.layers[0], None, None)
    with pytest.raises(NotImplementedError):
        RolloutEngine(cfg, "cpu", weight_dtype="fp8")


def test_extend_serves_llama_models_too():
    from polyrl_b200.models import TransformerWeights, get_model_config
    from polyrl_b200.models.transformer import PackedInput, forward_hidden, logits_forward
    from polyrl_b200.rollout.engine import RolloutEngine

    cfg = get_model_config("tiny-llama")
    w = TransformerWeights(cfg, seed=2)
    eng = RolloutEngine(cfg, "cpu", max_num_seqs=4, max_model_len=64)
    eng.set_weights(w.embed, w.layers, w.head)
    toks = {"a": seq(40, 512, 1), "b": seq(9, 512, 2)}
    got = feed(eng, toks, [[("a", 17), ("b", 3)], [("b", 1), ("a", 20)], [("a", 1), ("b", 1)], [("a", 2), ("b", 4)]])
    for k, t in toks.items():
        ids = torch.tensor(t)
        inp = PackedInput(ids, torch.arange(len(t)), torch.tensor([0, len(t)], dtype=torch.int32), len(t))
        want = logits_forward(cfg, w.head, w.embed, forward_hidden(cfg, w, inp))
        assert err(got[k], want.double()) < 1e-4


def test_odd_and_even_models_differ_from_their_parts():
    """The configurations above reach every branch: reused layers, a layer without feed-forward, grouped heads, unequal sizes."""
    assert any("weights_of" in x for x in ODD["layers"]) and any(x["mlp"] is None for x in ODD["layers"] + EVEN["layers"])
    assert MAMBA_EVEN["heads"] != MAMBA_EVEN["groups"] > 1
