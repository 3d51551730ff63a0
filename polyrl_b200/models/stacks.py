"""Designs built from the mixers of ``hybrid.py``: their ``config.json`` and their checkpoint names, both directions.

A design is one ``Design`` entry of ``DESIGNS``; ``ModelConfig.hf_model_type`` of a mixer stack is its key.  Checkpoint names start with
``l<i>.`` for layer ``i``; layers that reuse another's weights have no tensors.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Callable

import torch

from ..ops import reference as ref
from .config import ModelConfig
from .hybrid import gate_up_stacks, owner


@dataclass(frozen=True)
class Design:
    architecture: str
    kinds: dict                         # config.json mixer type -> layer kind
    read_layer: Callable                # (entry of config.json's layers, kind, index) -> {"sizes", "ff", ...}
    write_layer: Callable               # (layer of ModelConfig.layers) -> {"mixer", "mlp"}
    parts: Callable                     # (cfg, i) -> [(our name, [checkpoint names whose rows it stacks], [rows of each])]
    mlp_kinds: tuple = ("dense",)       # feed-forward kinds of config.json
    read_model: Callable = lambda hf: {}            # config.json -> further ModelConfig fields of the design
    write_model: Callable = lambda cfg: {}          # and back: further entries of config.json
    complete: Callable = lambda e, i, shape: e      # (entry of layers, index, name -> shape or None): sizes that only a tensor's shape tells


def sizes_from_tensors(hf: dict, folder) -> dict:
    """config.json with the sizes filled in that stand in no other place than the shapes of the folder's tensors."""
    from .hf_io import tensor_shape

    design = DESIGNS[hf["architecture"].lower()]
    return dict(hf, layers=[design.complete(e, i, lambda name: tensor_shape(folder, name)) for i, e in enumerate(hf["layers"])])


def stack_config(design: Design, hf: dict) -> ModelConfig:
    layers = []
    for i, e in enumerate(hf["layers"]):
        if e["type"] not in design.kinds:
            raise ValueError(f"{design.architecture} layer {i}: unknown mixer type {e['type']!r}")
        mlp = e.get("mlp")
        if mlp and mlp.get("kind", "dense") not in design.mlp_kinds:
            raise ValueError(f"{design.architecture} layer {i}: feed-forward kind {mlp['kind']!r}")
        kind = design.kinds[e["type"]]
        layers.append({"kind": kind, "ff": int(mlp.get("ff", 0)) if mlp else 0, "weights_of": int(e.get("weights_of", i)), **design.read_layer(e, kind, i)})
    return ModelConfig(family="hybrid", vocab_size=hf["vocab"], hidden_size=hf["width"], num_layers=len(layers), layers=tuple(layers),
                       intermediate_size=max([x["ff"] for x in layers] + [1]), num_heads=1, num_kv_heads=1, rms_norm_eps=float(hf["norm"]["eps"]),
                       eos_token_id=-1, bos_token_id=-1, pad_token_id=0, hf_model_type=design.architecture.lower(), name=design.architecture.lower(),
                       **design.read_model(hf))


def stack_config_dict(cfg: ModelConfig) -> dict:
    """``config.json`` of a stack (inverse of ``stack_config``)."""
    design = DESIGNS[cfg.hf_model_type]
    back = {v: k for k, v in design.kinds.items()}
    layers = []
    for i, lay in enumerate(cfg.layers):
        e = {"type": back[lay["kind"]], **design.write_layer(lay)}
        if lay["weights_of"] != i:
            e["weights_of"] = lay["weights_of"]
        layers.append(e)
    return {"architecture": design.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_norm_eps}, "layers": layers,
            **design.write_model(cfg)}


_MODEL_NAMES = {"embed": "embed", "norm_w": "final.norm", "lm_head": "head"}


def _map_gate_up(cfg: ModelConfig, i: int, t: dict, fn: Callable) -> None:
    """Replace every stack of gate and up rows of layer ``i`` by ``fn(rows)``, expert by expert, where the width has whole blocks of 128."""
    for name, count, width in gate_up_stacks(cfg.layers[i]):
        if width % 128 == 0:
            key = f"layers.{i}.{name}"
            t[key] = torch.cat([fn(x) for x in t[key].chunk(count)])


def stack_state_dict(cfg: ModelConfig, get) -> dict[str, torch.Tensor]:
    """Checkpoint -> our names; ``get`` reads a checkpoint tensor by name."""
    design = DESIGNS[cfg.hf_model_type]
    out = {n: get(s) for n, s in _MODEL_NAMES.items()}
    for i, lay in enumerate(cfg.layers):
        if owner(cfg, i) != i:
            continue
        p, q = f"l{i}.", f"layers.{i}."
        for n, names, _ in design.parts(cfg, i):
            out[q + n] = get(p + names[0]) if len(names) == 1 else torch.cat([get(p + s) for s in names])
        if design.kinds.get("mamba2") == lay["kind"]:            # one checkpoint tensor [in | step sizes] is two of ours
            w, nh = get(p + "mix.in"), lay["sizes"]["heads"]
            out[q + "w_in"], out[q + "w_dt"] = w[:-nh], w[-nh:]
        _map_gate_up(cfg, i, out, lambda x: ref.interleave_gate_up(*x.chunk(2)))
    return out


def stack_export(cfg: ModelConfig, sd: dict) -> dict[str, torch.Tensor]:
    """Our names -> checkpoint names (inverse of ``stack_state_dict``)."""
    design = DESIGNS[cfg.hf_model_type]
    sd = dict(sd)
    out = {s: sd[n] for n, s in _MODEL_NAMES.items()}
    for i, lay in enumerate(cfg.layers):
        if owner(cfg, i) != i:
            continue
        p, q = f"l{i}.", f"layers.{i}."
        _map_gate_up(cfg, i, sd, lambda x: torch.cat(ref.deinterleave_gate_up(x)))
        for n, names, rows in design.parts(cfg, i):
            t = sd[q + n]
            if len(names) == 1:
                out[p + names[0]] = t
            else:
                for s, piece in zip(names, t.split(rows)):
                    out[p + s] = piece.clone()
        if design.kinds.get("mamba2") == lay["kind"]:
            out[p + "mix.in"] = torch.cat([sd[q + "w_in"], sd[q + "w_dt"]])
    return out


def _one(ours: str, theirs: str) -> tuple[str, list[str], list[int]]:
    return ours, [theirs], []


# --------------------------------------------------------------------------------------------
# Ludesun: Mamba-2, xLSTM matrix memory and latent attention; RMS norms on the sublayer outputs, GELU feed-forward
# --------------------------------------------------------------------------------------------
_LUDESUN_SIZES = {"ssd": ("heads", "vdim", "state", "groups", "conv", "norm_groups"), "mlstm": ("heads", "dim", "vdim", "gate_cap"),
                  "latent": ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale")}


def _ludesun_read(e: dict, kind: str, i: int) -> dict:
    sizes = {k: e["mixer"][k] for k in _LUDESUN_SIZES[kind]}
    if kind == "latent":
        if e["mixer"]["rot"]["dims"] != sizes["rot_dim"]:
            raise ValueError(f"Ludesun layer {i}: rot.dims and rot_dim differ")
        sizes["rot_base"] = float(e["mixer"]["rot"]["base"])
    return {"sizes": sizes}


def _ludesun_write(lay: dict) -> dict:
    mx = {k: lay["sizes"][k] for k in _LUDESUN_SIZES[lay["kind"]]}
    if lay["kind"] == "latent":
        mx["rot"] = {"dims": mx["rot_dim"], "base": lay["sizes"]["rot_base"]}
    return {"mixer": mx, "mlp": {"kind": "dense", "ff": lay["ff"]} if lay["ff"] else None}


def _ludesun_parts(cfg: ModelConfig, i: int) -> list:
    lay = cfg.layers[i]
    m, h = lay["sizes"], lay["sizes"]["heads"]
    if lay["kind"] == "ssd":             # the input projection is split by the callers
        out = [_one("conv_w", "mix.conv"), _one("conv_b", "mix.conv.b"), _one("dt_bias", "mix.dt_bias"), _one("a_log", "mix.A_log"),
               _one("d_skip", "mix.D"), _one("gn", "mix.norm")]
    elif lay["kind"] == "mlstm":
        hd, hv = h * m["dim"], h * m["vdim"]
        out = [("w_in", ["mix.q", "mix.k", "mix.v", "mix.g"], [hd, hd, hv, hv]), ("w_if", ["mix.i", "mix.f"], [h, h]),
               ("b_if", ["mix.i.b", "mix.f.b"], [h, h]), _one("gn", "mix.norm")]
    else:
        out = [("wa", ["mix.dq", "mix.dkv"], [m["q_rank"], m["kv_rank"] + m["rot_dim"]]), _one("q_ln", "mix.dq.norm"), _one("kv_ln", "mix.dkv.norm"),
               _one("wq_up", "mix.uq"), _one("wk_up", "mix.uk"), _one("wv_up", "mix.uv"), _one("sink", "mix.sink")]
    out += [_one("wo", "mix.o"), _one("norm1", "norm1")]
    if lay["ff"]:
        out += [_one("norm2", "norm2"), _one("wup", "mlp.up"), _one("wdown", "mlp.down")]
    return out


# --------------------------------------------------------------------------------------------
# Lanilix: gated delta rule and windowed attention whose values are its keys; norms around every sublayer with weights stored around
# zero, clamped gated feed-forward
# --------------------------------------------------------------------------------------------
_LANILIX_SIZES = {"delta": ("heads", "kv_heads", "dim", "vdim", "conv"), "window": ("heads", "kv_heads", "dim", "vdim", "scale")}
_LANILIX_GLU_ALPHA = 1.702


def _lanilix_read(e: dict, kind: str, i: int) -> dict:
    m = e["mixer"]
    sizes = {k: m[k] for k in _LANILIX_SIZES[kind]}
    if kind == "window":
        sizes.update(window=int(m["mask"]["size"]), keep_first=int(m["mask"]["keep_first"]), rot_dim=int(m["rot"]["dims"]), rot_base=float(m["rot"]["base"]))
    out = {"sizes": sizes}
    if e.get("mlp"):
        out.update(act="clamped_glu", limit=float(e["mlp"]["limit"]), alpha=_LANILIX_GLU_ALPHA)
    return out


def _lanilix_write(lay: dict) -> dict:
    s = lay["sizes"]
    mx = {k: s[k] for k in _LANILIX_SIZES[lay["kind"]]}
    if lay["kind"] == "window":
        mx.update(mask={"size": s["window"], "keep_first": s["keep_first"]}, rot={"dims": s["rot_dim"], "base": s["rot_base"]})
    return {"mixer": mx, "mlp": {"kind": "dense", "ff": lay["ff"], "limit": lay["limit"]} if lay["ff"] else None}


def _lanilix_parts(cfg: ModelConfig, i: int) -> list:
    lay = cfg.layers[i]
    m, h, g = lay["sizes"], lay["sizes"]["heads"], lay["sizes"]["kv_heads"]
    qk, hv = g * m["dim"], h * m["vdim"]
    if lay["kind"] == "delta":
        out = [("w_in", ["mix.q", "mix.k", "mix.v", "mix.g"], [qk, qk, hv, hv]), ("w_ab", ["mix.a", "mix.b"], [h, h]),
               ("conv_w", ["mix.q.conv", "mix.k.conv", "mix.v.conv"], [qk, qk, hv]), _one("dt_bias", "mix.dt_bias"), _one("a_log", "mix.A_log"),
               _one("gn", "mix.norm")]
    else:
        out = [("wqk", ["mix.q", "mix.k"], [h * m["dim"], qk]), _one("q_norm", "mix.q.norm"), _one("k_norm", "mix.k.norm")]
    out += [_one("wo", "mix.o"), _one("pre1", "norm1"), _one("norm1", "norm1b")]
    if lay["ff"]:
        out += [_one("pre2", "norm2"), _one("norm2", "norm2b"), ("wgu", ["mlp.gate", "mlp.up"], [lay["ff"]] * 2), _one("wdown", "mlp.down")]
    return out


# --------------------------------------------------------------------------------------------
# experts
# --------------------------------------------------------------------------------------------
def _expert_parts(cfg: ModelConfig, lay: dict) -> list:
    n, f = lay["experts"], lay["ff"]
    out = [("ewgu", [f"mlp.e{j}.{k}" for j in range(n) for k in ("gate", "up")], [f] * (2 * n)),
           ("ewd", [f"mlp.e{j}.down" for j in range(n)], [cfg.hidden_size] * n), _one("router", "mlp.router")]
    if lay["shared"]:
        out += [("swgu", ["mlp.shared.gate", "mlp.shared.up"], [lay["shared"]] * 2), _one("swd", "mlp.shared.down")]
    return out


# --------------------------------------------------------------------------------------------
# Mabedra: differential attention in a sliding window; parallel blocks behind layer norms, with input convolutions, layer scales and
# averages over depth; dense layers with a polynomial activation, sparse ones with a sigmoid router and a shared expert
# --------------------------------------------------------------------------------------------
_MABEDRA_SIZES = ("heads", "kv_heads", "dim", "vdim", "scale", "diff")
_MABEDRA_MAPS = 2


def _mabedra_read(e: dict, kind: str, i: int) -> dict:
    m, mlp = e["mixer"], e.get("mlp")
    rot = m["rot"]
    sizes = {k: m[k] for k in _MABEDRA_SIZES}
    sizes.update(window=int(m["mask"]["size"]), rot_dim=int(rot["dims"]), rot_base=float(rot["base"]))
    if rot.get("scaling"):
        sizes["rot_scaling"] = {k: float(rot["scaling"][k]) for k in ("factor", "low", "high", "original")}
    out = {"sizes": sizes}
    if mlp and mlp["kind"] == "moe":
        out.update(act="moe", ff=int(mlp["expert"]["ff"]), experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]),
                   shared=int(mlp["shared"]["ff"]) if mlp.get("shared") else 0)
    elif mlp:
        out["act"] = "poly"
    return out


def _mabedra_write(lay: dict) -> dict:
    s, mlp = lay["sizes"], None
    mx = {k: s[k] for k in _MABEDRA_SIZES}
    mx.update(mask={"size": s["window"]}, rot={"dims": s["rot_dim"], "base": s["rot_base"]})
    if "rot_scaling" in s:
        mx["rot"]["scaling"] = dict(s["rot_scaling"])
    if lay["ff"] and lay["act"] == "moe":
        mlp = {"kind": "moe", "expert": {"ff": lay["ff"]}, "router": {"experts": lay["experts"], "top": lay["top"]}}
        if lay["shared"]:
            mlp["shared"] = {"ff": lay["shared"]}
    elif lay["ff"]:
        mlp = {"kind": "dense", "ff": lay["ff"]}
    return {"mixer": mx, "mlp": mlp}


def _mabedra_parts(cfg: ModelConfig, i: int) -> list:
    lay = cfg.layers[i]
    m, h, g, f = lay["sizes"], lay["sizes"]["heads"], lay["sizes"]["kv_heads"], lay["ff"]
    rows = [_MABEDRA_MAPS * h * m["dim"], _MABEDRA_MAPS * g * m["dim"], g * m["vdim"]]
    out = [("wqkv", ["mix.q", "mix.k", "mix.v"], rows), ("b_qkv", ["mix.q.b", "mix.k.b", "mix.v.b"], rows), _one("q_norm", "mix.q.norm"),
           _one("k_norm", "mix.k.norm"), ("map_mix", ["mix.lq1", "mix.lk1", "mix.lq2", "mix.lk2"], [m["dim"]] * 4), _one("wo", "mix.o"),
           _one("pre1", "norm1"), _one("ls1", "ls1"), _one("conv1", "canon1"), _one("depth", "dwa")]
    if not f:
        return out
    out += [_one("ls2", "ls2"), _one("conv2", "canon2")]
    if lay["act"] == "poly":
        return out + [_one("wup", "mlp.up"), _one("wdown", "mlp.down"), _one("act", "mlp.act")]
    return out + _expert_parts(cfg, lay)


# --------------------------------------------------------------------------------------------
# Dubazen: residual streams with hyper-connections; attention with rotated values beside linear attention with constant decays, gated linear
# attention, selective scans; clamped experts behind a softmax router.  The rank of a gla layer's decay is told by its tensors only.
# --------------------------------------------------------------------------------------------
_DUBAZEN_SIZES = {"selective": ("inner", "state", "dt_rank", "conv"), "gla": ("heads", "dim", "vdim", "tau"), "turn": ("heads", "kv_heads", "dim", "vdim", "scale"),
                  "decay": ("heads", "dim", "vdim")}
_DUBAZEN_GLU_ALPHA = 1.702


def _dubazen_complete(e: dict, i: int, shape: Callable) -> dict:
    if e["type"] != "gla" or "rank" in e["mixer"]:
        return e
    found = shape(f"l{i}.mix.a1")
    return e if found is None else dict(e, mixer=dict(e["mixer"], rank=found[0]))


def _dubazen_read(e: dict, kind: str, i: int) -> dict:
    m, mlp = e["mixer"], e.get("mlp")
    if kind == "pair":
        a, r = m["left"], m["right"]
        sizes = {"left": {"kind": "turn", **{k: a[k] for k in _DUBAZEN_SIZES["turn"]}, "rot_dim": int(a["rot"]["dims"]), "rot_base": float(a["rot"]["base"])},
                 "right": {"kind": "decay", **{k: r[k] for k in _DUBAZEN_SIZES["decay"]}, "decay": [float(x) for x in r["decay"]]},
                 "left_scale": float(m["left_scale"]), "right_scale": float(m["right_scale"])}
    else:
        sizes = {k: m[k] for k in _DUBAZEN_SIZES[kind]}
        if kind == "gla":
            if "rank" not in m:
                raise ValueError(f"Dubazen layer {i}: the rank of the decay is told by the model's tensors (or by mixer.rank)")
            sizes["rank"] = int(m["rank"])
    out = {"sizes": sizes}
    if mlp:
        shared = mlp.get("shared")
        out.update(act="moe", router="softmax", ff=int(mlp["expert"]["ff"]), experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]),
                   shared=int(shared["ff"]) if shared else 0, limit=float(mlp["expert"]["limit"]), shared_limit=float(shared["limit"]) if shared else 0.0,
                   alpha=_DUBAZEN_GLU_ALPHA)
    return out


def _dubazen_write(lay: dict) -> dict:
    s, mlp = lay["sizes"], None
    if lay["kind"] == "pair":
        a, r = s["left"], s["right"]
        mx = {"left": {**{k: a[k] for k in _DUBAZEN_SIZES["turn"]}, "rot": {"dims": a["rot_dim"], "base": a["rot_base"]}},
              "right": {**{k: r[k] for k in _DUBAZEN_SIZES["decay"]}, "decay": list(r["decay"])}, "left_scale": s["left_scale"], "right_scale": s["right_scale"]}
    else:
        mx = {k: s[k] for k in _DUBAZEN_SIZES[lay["kind"]]}
    if lay["ff"]:
        mlp = {"kind": "moe", "expert": {"ff": lay["ff"], "limit": lay["limit"]}, "router": {"experts": lay["experts"], "top": lay["top"]}}
        if lay["shared"]:
            mlp["shared"] = {"ff": lay["shared"], "limit": lay["shared_limit"]}
    return {"mixer": mx, "mlp": mlp}


def _dubazen_parts(cfg: ModelConfig, i: int) -> list:
    lay = cfg.layers[i]
    m, kind = lay["sizes"], lay["kind"]
    if kind == "pair":
        a, r = m["left"], m["right"]
        rows = [a["heads"] * a["dim"], a["kv_heads"] * a["dim"], a["kv_heads"] * a["vdim"]]
        out = [("left.w_in", [f"mix.left.{n}" for n in "qkvg"], rows + [a["heads"] * a["vdim"]]), ("left.b_qkv", [f"mix.left.{n}.b" for n in "qkv"], rows),
               _one("left.sink", "mix.left.sink"), _one("left.wo", "mix.left.o"), _one("left.b_o", "mix.left.o.b"),
               ("right.w_in", [f"mix.right.{n}" for n in "qkvg"], [r["heads"] * r["dim"]] * 2 + [r["heads"] * r["vdim"]] * 2), _one("right.gn", "mix.right.norm"),
               _one("right.wo", "mix.right.o")]
    elif kind == "gla":
        out = [("w_in", ["mix.q", "mix.k", "mix.v", "mix.g", "mix.a1"], [m["heads"] * m["dim"]] * 2 + [m["heads"] * m["vdim"]] * 2 + [m["rank"]]),
               _one("w_a", "mix.a2"), _one("b_a", "mix.a2.b"), _one("gn", "mix.norm"), _one("wo", "mix.o")]
    else:
        out = [_one("w_in", "mix.in"), _one("conv_w", "mix.conv"), _one("conv_b", "mix.conv.b"), _one("w_x", "mix.x"), _one("w_dt", "mix.dt"),
               _one("dt_bias", "mix.dt.b"), _one("a_log", "mix.A_log"), _one("d_skip", "mix.D"), _one("wo", "mix.o")]
    for q in ("1", "2") if lay["ff"] else ("1",):
        out += [_one("pre" + q, "norm" + q)] + [_one(f"hc{q}.{n}", f"hc{q}.{n}") for n in ("in", "out", "mix")]
    return out + (_expert_parts(cfg, lay) if lay["ff"] else [])


DESIGNS = {
    "ludesun": Design("Ludesun", {"mamba2": "ssd", "mlstm": "mlstm", "latent_attention": "latent"}, _ludesun_read, _ludesun_write, _ludesun_parts),
    "lanilix": Design("Lanilix", {"delta": "delta", "attention": "window"}, _lanilix_read, _lanilix_write, _lanilix_parts,
                      read_model=lambda hf: {"sandwich_norm": True, "norm_offset": 1.0}),
    "mabedra": Design("Mabedra", {"attention": "diff"}, _mabedra_read, _mabedra_write, _mabedra_parts, mlp_kinds=("dense", "moe"),
                      read_model=lambda hf: {"parallel_block": True, "layer_norm": True, "layer_scale": True, "depth_average": True,
                                             "input_conv": int(hf["canon"]["taps"])},
                      write_model=lambda cfg: {"canon": {"taps": cfg.input_conv}}),
    "dubazen": Design("Dubazen", {"parallel": "pair", "gla": "gla", "mamba1": "selective"}, _dubazen_read, _dubazen_write, _dubazen_parts, mlp_kinds=("moe",),
                      read_model=lambda hf: {"streams": int(hf["streams"]), "scalar_norm": True, "embed_scale": float(hf["embedding"]["scale"])},
                      write_model=lambda cfg: {"streams": cfg.streams, "embedding": {"scale": cfg.embed_scale}}, complete=_dubazen_complete),
}
