"""Dubazen stacks through the framework's configuration, loader, scheduler, cache / state manager and step functions, on CPU in fp32, against the
plain oracle (tests/dubazen_oracle.py)."""
import io
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(__file__))
import dubazen_oracle as oracle                       # noqa: E402
from dubazen_util import CONFIGS, P_EVEN, P_ODD, cut, decay, err, feed, gla, layer, make_engine, mamba, model, moe, pair, reference, seq, turn   # noqa: E402

TOL = 1e-4


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, cfg in CONFIGS.items():
        sd = oracle.random_model(cfg, seed=len(name), gla_rank={"odd": 3, "even": 8, "one": 1}[name])
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
ALONE = {"pair": P_ODD, "pair-even": P_EVEN, "pair-heads": pair(turn(4, 4, 6, 4, 6), decay(1, 16, 8, (0.3,)), 0.0, 1.0), "left": pair(turn(6, 3, 9, 8, 2), decay(3, 4, 4, (0.0, 0.5, 1.0)), 1.0, 0.0),
         "gla": gla(4, 8, 12, 16.0), "gla-fast": gla(2, 5, 7, 0.3), "mamba": mamba(30, 6, 4, 3), "mamba-plain": mamba(16, 1, 7, 1), "mamba-wide": mamba(8, 40, 2, 2)}


@pytest.mark.parametrize("name", list(ALONE))
def test_mixers_alone(tmp_path, name):
    cfg = model(40, 50, layer(ALONE[name]), streams=2)
    sd = oracle.random_model(cfg, 5, gla_rank=6)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(80, 50, 9), "b": seq(33, 50, 10)}
    got = feed(make_engine(tmp_path / "m"), toks, [[("a", 50), ("b", 16)], [("a", 1), ("b", 15)], [("a", 28), ("b", 1)], [("b", 1), ("a", 1)]])
    want = reference(cfg, sd, toks)
    assert max(err(got[k], want[k]) for k in toks) < TOL


def test_every_tensor_matters(folders):
    """The oracle's logits move with each kind of tensor: what follows is able to see a fault in any of them."""
    for name in ("odd", "even"):
        cfg, sd, _ = folders[name]
        t = seq(25, cfg["vocab"], 1)
        base = oracle.forward(cfg, sd, t)
        for k in sd:
            if ".e" in k or k.endswith("router") or k == "l0.hc1.in":              # (equal streams: only the sum of "in" counts, and the norm divides it out)
                continue
            other = dict(sd, **{k: sd[k] * 1.5 + 0.1})
            assert err(oracle.forward(cfg, other, t), base) > (1e-6 if k.endswith("k.b") else 1e-4), k


def far_model(sink=-40.0, rate=None):
    """One attention layer in which token 1 asks and token 2 is the key that answers, its score standing out by e^8; every other pair scores zero."""
    d = 8
    cfg = model(16, 12, layer(pair(turn(1, 1, d, 8, 2, 100.0, 1.0), decay(1, 2, 2, (0.5,)), 1.0, 0.0)), streams=2, scale=1.0)
    sd = oracle.random_model(cfg, 11)
    e = torch.zeros(12, 16, dtype=oracle.D)
    for t in range(12):
        e[t, t] = 4.0
    sd["embed"] = e
    for n, v in (("in", [0.5, 0.5]), ("out", [1.0, 1.0])):
        sd[f"l0.hc1.{n}"] = torch.tensor(v, dtype=oracle.D)
    sd["l0.hc1.mix"], sd["l0.norm1"] = torch.eye(2, dtype=oracle.D), torch.tensor(1.0, dtype=oracle.D)
    q, k = torch.zeros(d, 16, dtype=oracle.D), torch.zeros(d, 16, dtype=oracle.D)
    q[2, 1] = q[3, 5] = 4.0                                        # the rotation turns entries 0 and 1 only
    k[2, 2] = 4.0
    for t in [x for x in range(12) if x != 2]:
        k[4 + t % 4, t] = 4.0
    sd["l0.mix.left.q"], sd["l0.mix.left.k"] = q, k
    for n in ("q.b", "k.b", "v.b"):
        sd[f"l0.mix.left.{n}"] = torch.zeros_like(sd[f"l0.mix.left.{n}"])
    sd["l0.mix.left.sink"] = torch.full((1,), sink, dtype=oracle.D)
    return cfg, {k: t.to(torch.bfloat16).to(oracle.D) for k, t in sd.items()}


def test_keys_far_away_and_at_page_borders(tmp_path):
    cfg, sd = far_model()
    oracle.write_model(cfg, sd, tmp_path / "m")
    for at in (0, 1, 15, 16, 31, 32):
        t = [4 + x for x in seq(100, 8, at)]
        t[at] = 2
        asks = [at + 1, at + 2, 47, 48, 98, 99]
        for q in asks:
            t[q] = 1
        want = reference(cfg, sd, {"a": t})["a"]
        hidden = list(t)
        hidden[at] = 4                                             # the same sequence without that key
        diff = (reference(cfg, sd, {"a": hidden})["a"] - want).pow(2).mean(-1).sqrt()
        assert all(diff[q] > 0.02 for q in asks)
        for steps in ([100], cut(100, (33, 16, 1)), cut(100, (2,)), [at + 1] + [1] * (99 - at)):
            assert err(feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in steps])["a"], want) < TOL, (at, steps)


@pytest.mark.parametrize("sink", [-40.0, 0.0, 3.0, 9.0])
def test_sink_counts_once_and_unscaled(tmp_path, sink):
    cfg, sd = far_model(sink)
    cfg["layers"][0]["mixer"]["left"]["scale"] = 0.5
    oracle.write_model(cfg, sd, tmp_path / "m")
    t = [2] + [4 + x for x in seq(40, 8, 3)] + [1]
    want = oracle.forward(cfg, sd, t)
    if sink > 0:
        for other in (-40.0, sink * 0.5, sink + math.log(2)):
            assert err(oracle.forward(cfg, dict(sd, **{"l0.mix.left.sink": torch.full((1,), other, dtype=oracle.D)}), t), want) > 1e-3
    for sizes in ((42,), (1,), (17, 2)):
        assert err(feed(make_engine(tmp_path / "m"), {"a": t}, [[("a", n)] for n in cut(42, sizes)])["a"], want) < TOL


def test_values_are_rotated_and_outputs_turned_back():
    """Only the distance counts: the output moves with a sequence's place only through what the keys see."""
    from polyrl_b200.ops import mixers as M

    H, G, d, e, T = 4, 2, 6, 10, 9
    g = torch.Generator().manual_seed(0)
    p = torch.randn(T, (H + G) * d + G * e, generator=g)
    gate = torch.randn(T, H * e, generator=g)
    outs = []
    for at in (0, 37):
        b = M.SpanBatch(cu=torch.tensor([0, T], dtype=torch.int32), start=torch.tensor([0], dtype=torch.int32), slot=torch.zeros(1, dtype=torch.long), pos=torch.arange(T) + at,
                        kv_slot=16 + torch.arange(T), kv_len=torch.arange(1, T + 1, dtype=torch.int32), table=torch.tensor([[1, 2]], dtype=torch.int32),
                        seq_of=torch.zeros(T, dtype=torch.int32), n_long=1, t_long=T, max_long=T, max_len=T)
        kp, vp = torch.zeros(4, G, 16, d), torch.zeros(4, G, 16, e)
        vf = M.rope_frequencies(e, 50.0, "cpu")
        q, _ = M.turn_prep(p, torch.zeros(p.shape[1]), H, d, e, M.rope_frequencies(4, 50.0, "cpu"), vf, kp, vp, b, 1e-6, False)
        o = M.sink_attention(q, kp, vp, b.table, b.seq_of, b.kv_len, 0.7, torch.zeros(H), T)
        outs.append(M.turn_back(o, gate, vf, b.pos, 1.0, torch.empty(T, H * e)))
    assert (outs[0] - outs[1]).abs().max() < 1e-5 and outs[0].abs().max() > 0.1


@pytest.mark.parametrize("n,top,ff,shared", [(5, 2, 24, 7), (4, 4, 128, 16), (9, 1, 7, 130), (1, 1, 8, 8), (40, 6, 5, 3)])
def test_experts_alone(tmp_path, n, top, ff, shared):
    cfg = model(32, 40, layer(mamba(4, 1, 1, 1), moe(n, top, ff, shared)), streams=2)
    sd = oracle.random_model(cfg, n)
    for k in sd:
        if ".mlp." in k:
            sd[k] = ((0.5 if k.endswith("router") else 2) * sd[k]).to(torch.bfloat16).to(oracle.D)
    oracle.write_model(cfg, sd, tmp_path / "m")
    toks = {"a": seq(40, 40, 1)}
    want = reference(cfg, sd, toks)["a"]
    assert err(feed(make_engine(tmp_path / "m"), toks, [[("a", 25)], [("a", 1)], [("a", 14)]])["a"], want) < TOL
    for part in ("expert", "shared"):                              # both limits bite
        other = json.loads(json.dumps(cfg))
        other["layers"][0]["mlp"][part]["limit"] = 30.0
        assert err(oracle.forward(other, sd, toks["a"]), want) > 1e-3


def test_streams(tmp_path):
    """Maps that are neither symmetric nor alike: from and to, both sublayers, one stream and many."""
    for n in (1, 2, 7):
        cfg = model(24, 30, layer(mamba(10, 2, 2, 2), moe(2, 1, 8, 8)), layer(gla(1, 4, 4, 2.0)), layer(mamba(10, 2, 2, 2), moe(2, 1, 8, 8)), streams=n, scale=0.3)
        sd = oracle.random_model(cfg, n, gla_rank=2)
        g = torch.Generator().manual_seed(n)
        for k in sd:
            if ".hc" in k:
                sd[k] = (torch.randn(sd[k].shape, generator=g) * n ** -0.5 + (1 if n == 1 else 0)).to(torch.bfloat16).to(oracle.D)
        oracle.write_model(cfg, sd, tmp_path / str(n))
        t = seq(20, 30, 3)
        want = oracle.forward(cfg, sd, t)
        if n > 1:
            assert err(oracle.forward(cfg, {k: x.T if k.endswith(".mix") and "hc" in k else x for k, x in sd.items()}, t), want) > 1e-2
        for sizes in ((20,), (1,), (3, 2)):
            assert err(feed(make_engine(tmp_path / str(n)), {"a": t}, [[("a", x)] for x in cut(20, sizes)])["a"], want) < TOL


def test_long_decoding_keeps_slow_states(tmp_path):
    cfg = model(16, 20, layer(pair(turn(1, 1, 4, 4, 2), decay(2, 4, 4, (0.999, 0.9999)), 0.2, 1.0)), layer(gla(1, 4, 4, 16.0)), layer(mamba(8, 3, 2, 3)), streams=2)
    sd = oracle.random_model(cfg, 2, gla_rank=2)
    sd["l1.mix.a2.b"] = torch.full((4,), 5.0, dtype=oracle.D)
    oracle.write_model(cfg, sd, tmp_path / "m")
    t = seq(400, 20, 4)
    want = oracle.forward(cfg, sd, t)
    other = [(t[0] + 1) % 20] + t[1:]
    assert (oracle.forward(cfg, sd, other)[-1] - want[-1]).abs().max() > 1e-4           # the first token is still there at the end
    assert err(feed(make_engine(tmp_path / "m", max_len=512, tokens=512), {"a": t}, [[("a", 5)]] + [[("a", 1)]] * 395)["a"], want) < TOL


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
    want = [greedy_oracle(cfg, sd, p, 8) for p in prompts]
    eng = make_engine(d, seqs=3, max_len=64, max_prefill_tokens=chunk)           # five requests through three slots
    for _ in range(2):
        out = eng.generate(prompts, dict(max_new_tokens=8, temperature=0.0))
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
    want = greedy_oracle(cfg, sd, prompt, 8)
    out = make_engine(d, seqs=4, max_len=64).generate([prompt], dict(max_new_tokens=8, temperature=0.0, n=3))
    assert [r.output_ids for r in out[0]] == [want] * 3


def test_config_registry_loader_and_export_round_trip(folders, tmp_path):
    from polyrl_b200.models import ModelConfig, get_model_config
    from polyrl_b200.models.hf_io import load_state_dict, save_hf

    for name in CONFIGS:
        cfg, sd, d = folders[name]
        mc = get_model_config(str(d))
        assert (mc.family, mc.num_layers, mc.vocab_size, mc.hidden_size) == ("hybrid", len(cfg["layers"]), cfg["vocab"], cfg["width"])
        assert mc.streams == cfg["streams"] and mc.embed_scale == cfg["embedding"]["scale"] and mc.num_params() == sum(t.numel() for t in sd.values())
        assert ModelConfig(**json.loads(json.dumps(mc.to_dict()))) == mc
        save_hf(load_state_dict(mc, d), mc, tmp_path / name)
        back = oracle.read_safetensors(tmp_path / name / "model.safetensors")
        assert set(back) == set(sd) and all(torch.equal(back[k], sd[k]) and back[k].shape == sd[k].shape for k in sd)
        assert get_model_config(str(tmp_path / name)) == mc
    cfg = folders["even"][0]
    first, second, third = cfg["layers"][:3]
    with pytest.raises(ValueError, match="rank"):                  # a config.json without its tensors
        ModelConfig.from_hf_config(cfg)
    second = dict(second, mixer=dict(second["mixer"], rank=8))
    assert ModelConfig.from_hf_config(dict(cfg, layers=[first, second, third])).layers[1]["sizes"]["rank"] == 8
    for bad in ([dict(first, type="conv")], [dict(first, mlp=dict(kind="dense", ff=8))], [dict(first, mlp=moe(3, 4, 8, 8))],
                [dict(first, mixer=dict(first["mixer"], state=600))], [dict(second, mixer=dict(second["mixer"], tau=0.0))],
                [dict(third, mixer=dict(third["mixer"], left=turn(3, 2, 4, 4, 2)))], [dict(third, mixer=dict(third["mixer"], right=decay(2, 4, 4, (0.5,))))],
                [dict(third, mixer=dict(third["mixer"], left=turn(2, 2, 4, 5, 2)))]):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_config(dict(cfg, layers=bad))
    with pytest.raises(ValueError):
        ModelConfig.from_hf_config(dict(cfg, layers=[first], streams=17))


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
        want = reference(cfg, sd, toks)["a"]
        assert ((got - want).pow(2).mean(-1).sqrt() / want.std()).median() < 0.1


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


def test_parts_in_other_stacks():
    """Streams, mixers and experts are independent of the design: vector norms and other mixers over streams, the new mixers in plain and parallel
    blocks, a softmax router behind a silu gate."""
    from polyrl_b200.models import ModelConfig, TransformerWeights
    from polyrl_b200.rollout.engine import RolloutEngine

    delta = dict(kind="delta", sizes=dict(heads=2, kv_heads=1, dim=6, vdim=5, conv=3), ff=24, act="gelu")
    att = dict(kind="turn", sizes=dict(heads=2, kv_heads=1, dim=6, vdim=4, scale=0.4, rot_dim=4, rot_base=100.0), ff=0)
    lin = dict(kind="decay", sizes=dict(heads=2, dim=6, vdim=4, decay=[0.5, 0.99]), ff=16, act="gelu")
    sparse = dict(kind="gla", sizes=dict(heads=2, dim=4, vdim=4, tau=2.0, rank=3), ff=16, act="moe", experts=4, top=2, shared=0, router="softmax")
    base = dict(family="hybrid", vocab_size=40, hidden_size=24, intermediate_size=24, num_heads=1, num_kv_heads=1, hf_model_type="", eos_token_id=-1)
    toks = {"a": seq(30, 40, 1)}
    for layers, kw in (((delta, att, lin, sparse), dict(streams=2)), ((att, lin), {}), ((att, lin), dict(sandwich_norm=True)), ((sparse, att, lin), dict(parallel_block=True))):
        cfg = ModelConfig(**base, num_layers=len(layers), layers=tuple(dict(x, weights_of=i) for i, x in enumerate(layers)), **kw)
        w = TransformerWeights(cfg, seed=1)
        outs = []
        for sizes in ((30,), (7, 1, 2)):
            eng = RolloutEngine(cfg, "cpu", max_num_seqs=2, max_model_len=64)
            eng.set_weights(w.embed, w.layers, w.head)
            outs.append(feed(eng, toks, [[("a", n)] for n in cut(30, sizes)])["a"])
        assert torch.isfinite(outs[0]).all() and err(outs[1], outs[0]) < TOL
    for bad in (dict(streams=2, parallel_block=True), dict(scalar_norm=True), dict(streams=2, sandwich_norm=True)):
        with pytest.raises(ValueError):
            ModelConfig(**base, num_layers=1, layers=(dict(delta, weights_of=0),), **bad)


def test_weight_updates_in_place(folders):
    """A second set of weights overwrites what was derived from the first: captured steps keep their addresses."""
    from polyrl_b200.models import TransformerWeights, get_model_config
    from polyrl_b200.models.hf_io import load_state_dict
    from polyrl_b200.rollout.engine import RolloutEngine

    cfg, sd, d = folders["even"]
    mc = get_model_config(str(d))
    eng = RolloutEngine(mc, "cpu", max_num_seqs=2, max_model_len=64, dtype=torch.float32)
    w = TransformerWeights(mc, dtype=torch.float32, seed=3)
    eng.set_weights(w.embed, w.layers, w.head)
    before = [{k: t.data_ptr() for k, t in x.items()} for x in eng.layer_w]
    w.load_state_dict({k: t.float() for k, t in load_state_dict(mc, d).items()})
    eng.set_weights(w.embed, w.layers, w.head)
    assert before == [{k: t.data_ptr() for k, t in x.items()} for x in eng.layer_w]
    toks = {"a": seq(12, cfg["vocab"], 2)}
    assert err(feed(eng, toks, [[("a", 12)]])["a"], reference(cfg, sd, toks)["a"]) < TOL


def test_presets():
    from polyrl_b200.models import TransformerWeights, get_model_config
    from polyrl_b200.rollout.engine import RolloutEngine

    cfg = get_model_config("tiny-dubazen")
    w = TransformerWeights(cfg, seed=1)
    assert cfg.num_params() == sum(t.numel() for _, t in w.named_tensors())
    assert w.layers[0]["pre1"].shape == () and (w.layers[0]["hc1.mix"] == torch.eye(3)).all() and (w.layers[1]["hc2.out"] == 1).all()
    eng = RolloutEngine(cfg, "cpu", max_num_seqs=2, max_model_len=32)
    eng.set_weights(w.embed, w.layers, w.head)
    assert len(eng.generate([[3, 4, 5]], dict(max_new_tokens=4, temperature=1.0))[0][0].output_ids) == 4
    assert get_model_config("dubazen-7b").num_params() > 6e9
