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
from .hybrid import owner


@dataclass(frozen=True)
class Design:
    architecture: str
    kinds: dict                         # config.json mixer type -> layer kind
    read_layer: Callable                # (entry of config.json's layers, kind, index) -> {"sizes", "ff", ...}
    write_layer: Callable               # (layer of ModelConfig.layers) -> {"mixer", "mlp"}
    parts: Callable                     # (cfg, i) -> [(our name, [checkpoint names whose rows it stacks], [rows of each])]
    glu: bool = False                   # feed-forward is gate / up / down
    model_fields: dict = None           # further ModelConfig fields of the design


def stack_config(design: Design, hf: dict) -> ModelConfig:
    layers = []
    for i, e in enumerate(hf["layers"]):
        if e["type"] not in design.kinds:
            raise ValueError(f"{design.architecture} layer {i}: unknown mixer type {e['type']!r}")
        mlp = e.get("mlp")
        if mlp and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"{design.architecture} layer {i}: feed-forward kind {mlp['kind']!r}")
        kind = design.kinds[e["type"]]
        layers.append({"kind": kind, "ff": int(mlp["ff"]) if mlp else 0, "weights_of": int(e.get("weights_of", i)), **design.read_layer(e, kind, i)})
    return ModelConfig(family="hybrid", vocab_size=hf["vocab"], hidden_size=hf["width"], num_layers=len(layers), layers=tuple(layers),
                       intermediate_size=max([x["ff"] for x in layers] + [1]), num_heads=1, num_kv_heads=1, rms_norm_eps=float(hf["norm"]["eps"]),
                       eos_token_id=-1, bos_token_id=-1, pad_token_id=0, hf_model_type=design.architecture.lower(), name=design.architecture.lower(),
                       **(design.model_fields or {}))


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
    return {"architecture": design.architecture, "vocab": cfg.vocab_size, "width": cfg.hidden_size, "norm": {"eps": cfg.rms_norm_eps}, "layers": layers}


_MODEL_NAMES = {"embed": "embed", "norm_w": "final.norm", "lm_head": "head"}


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
        if design.glu and lay["ff"] and lay["ff"] % 128 == 0:
            f = lay["ff"]
            out[q + "wgu"] = ref.interleave_gate_up(out[q + "wgu"][:f], out[q + "wgu"][f:])
    return out


def stack_export(cfg: ModelConfig, sd: dict) -> dict[str, torch.Tensor]:
    """Our names -> checkpoint names (inverse of ``stack_state_dict``)."""
    design = DESIGNS[cfg.hf_model_type]
    out = {s: sd[n] for n, s in _MODEL_NAMES.items()}
    for i, lay in enumerate(cfg.layers):
        if owner(cfg, i) != i:
            continue
        p, q = f"l{i}.", f"layers.{i}."
        for n, names, rows in design.parts(cfg, i):
            t = sd[q + n]
            if n == "wgu" and lay["ff"] % 128 == 0:
                t = torch.cat(ref.deinterleave_gate_up(t))
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


DESIGNS = {
    "ludesun": Design("Ludesun", {"mamba2": "ssd", "mlstm": "mlstm", "latent_attention": "latent"}, _ludesun_read, _ludesun_write, _ludesun_parts),
    "lanilix": Design("Lanilix", {"delta": "delta", "attention": "window"}, _lanilix_read, _lanilix_write, _lanilix_parts, glu=True,
                      model_fields={"sandwich_norm": True, "norm_offset": 1.0}),
}
