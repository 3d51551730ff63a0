"""Plain, slow oracle of the Mabedra design: whole sequences, double precision.  One function per mechanism; nothing here is shared with
the product path."""
import json
import math
import struct

import numpy as np
import torch

D = torch.float64


def read_safetensors(path):
    raw = open(path, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    out = {}
    for name, e in json.loads(raw[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if e["dtype"] == "BF16":
            t = torch.from_numpy((np.frombuffer(buf, np.uint16).astype(np.uint32) << 16).view(np.float32).copy())
        else:
            t = torch.from_numpy(np.frombuffer(buf, {"F32": np.float32, "I32": np.int32}[e["dtype"]]).copy())
        out[name] = t.reshape(e["shape"]).to(D)
    return out


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def silu(z):
    return z / (1 + torch.exp(-z))


def input_conv(h, w):
    """h + causal convolution of h per channel: w [C, taps], last column the current token, zeros before the sequence."""
    T, taps = h.shape[0], w.shape[1]
    y = h.clone()
    for t in range(T):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                y[t] = y[t] + w[:, j] * h[s]
    return y


def frequencies(rot):
    """Rotation speeds with long wavelengths slowed down (the three ranges of Llama 3.1)."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot["scaling"]
        turns = s["original"] * f / (2 * math.pi)                  # original length / wavelength
        if turns > s["high"]:
            g = f
        elif turns < s["low"]:
            g = f / s["factor"]
        else:
            a = (turns - s["low"]) / (s["high"] - s["low"])
            g = (1 - a) * f / s["factor"] + a * f
        out.append(g)
    return out


def rotate_half(x, freqs):
    """x [T, heads, maps, d]: entries (i, i + n) of the first 2 n turned by position * freqs[i]."""
    y, n = x.clone(), len(freqs)
    pos = torch.arange(x.shape[0], dtype=x.dtype)[:, None, None]
    for i, f in enumerate(freqs):
        u, v = x[..., i], x[..., i + n]
        c, s = torch.cos(pos * f), torch.sin(pos * f)
        y[..., i], y[..., i + n] = u * c - v * s, v * c + u * s
    return y


def visible(i, j, size):
    return 0 <= i - j < size


def map_attention(q, k, v, scale, size):
    """One map: q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]."""
    T, H = q.shape[:2]
    r = H // k.shape[1]
    seen = torch.tensor([[visible(i, j, size) for j in range(T)] for i in range(T)])
    o = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // r].T) * scale
        o[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, h // r]
    return o


def weight_of_second_map(w, diff):
    return torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + diff


def difference(a1, a2, lam, diff, eps):
    return rms(a1 - lam * a2, eps) * (1 - diff)


def attention(h, w, m, eps):
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    fr = frequencies(m["rot"])
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, 2, d)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, 2, d)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, e)
    q, k = rotate_half(rms(q, eps) * w["q.norm"], fr), rotate_half(rms(k, eps) * w["k.norm"], fr)
    a = [map_attention(q[:, :, i], k[:, :, i], v, m["scale"], m["mask"]["size"]) for i in range(2)]
    o = difference(a[0], a[1], weight_of_second_map(w, m["diff"]), m["diff"], eps)
    return o.reshape(T, H * e) @ w["o"].T


def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def gated(x, w, name):
    return (silu(x @ w[name + "gate"].T) * (x @ w[name + "up"].T)) @ w[name + "down"].T


def route(h, router, top):
    """[(experts, weights)] of every token: the largest sigmoid scores, as they are."""
    s = 1 / (1 + torch.exp(-(h @ router.T)))
    order = torch.argsort(s, dim=-1, descending=True)[:, :top]
    return order, s.gather(1, order)


def mixture(h, w, mlp):
    pick, weight = route(h, w["router"], mlp["router"]["top"])
    y = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in zip(pick[t].tolist(), weight[t]):
            y[t] += gated(g * h[t], w, f"e{e}.")
    return y + gated(h, w, "shared.") if mlp.get("shared") else y


def feed_forward(h, w, mlp, eps):
    if mlp["kind"] == "dense":
        return poly_norm(h @ w["up"].T, w["act"], eps) @ w["down"].T
    return mixture(h, w, mlp)


def forward(cfg, sd, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence (config.json dict, tensors by name)."""
    eps = cfg["norm"]["eps"]
    past = [sd["embed"][torch.as_tensor(tokens)]]
    x = past[0]
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = {part: {k[len(p) + 4:]: t for k, t in sd.items() if k.startswith(p + part + ".")} for part in ("mix", "mlp")}
        h = layer_norm(x, sd[p + "norm1"], eps)
        y = attention(input_conv(h, sd[p + "canon1"]), sub["mix"], lay["mixer"], eps) * sd[p + "ls1"]
        if lay.get("mlp"):
            y = y + feed_forward(input_conv(h, sd[p + "canon2"]), sub["mlp"], lay["mlp"], eps) * sd[p + "ls2"]
        past.append(x + y)
        x = sum(a * t for a, t in zip(sd[p + "dwa"], past))
        if layers_out is not None:
            layers_out.append(x)
    return layer_norm(x, sd["final.norm"], eps) @ sd["head"].T


def tensor_shapes(cfg):
    """Names and shapes of every tensor of a model folder."""
    W, out, taps = cfg["width"], {}, cfg["canon"]["taps"]
    out["embed"] = (cfg["vocab"], W)
    for i, lay in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lay["mixer"], lay.get("mlp")
        q = p + "mix."
        H, G, d, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        out.update({p + "norm1": (W,), p + "ls1": (W,), p + "canon1": (W, taps), p + "dwa": (i + 2,)})
        for n, rows in (("q", 2 * H * d), ("k", 2 * G * d), ("v", G * V)):
            out[q + n], out[q + n + ".b"] = (rows, W), (rows,)
        out.update({q + n: (d,) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
        out[q + "o"] = (W, H * V)
        if not mlp:
            continue
        out.update({p + "ls2": (W,), p + "canon2": (W, taps)})
        q = p + "mlp."
        if mlp["kind"] == "dense":
            out.update({q + "up": (mlp["ff"], W), q + "down": (W, mlp["ff"]), q + "act": (4,)})
            continue
        n = mlp["router"]["experts"]
        out[q + "router"] = (n, W)
        for name, F in [(f"e{j}", mlp["expert"]["ff"]) for j in range(n)] + ([("shared", mlp["shared"]["ff"])] if mlp.get("shared") else []):
            out.update({f"{q}{name}.gate": (F, W), f"{q}{name}.up": (F, W), f"{q}{name}.down": (W, F)})
    out["final.norm"], out["head"] = (W,), (cfg["vocab"], W)
    return out


def random_model(cfg, seed=0):
    """Random bf16-representable weights, spread enough that every one of them matters."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shp in tensor_shapes(cfg).items():
        t = torch.randn(shp, generator=g)
        base = name.split("mix.")[-1] if "mix." in name else name.split(".")[-1]
        if base in ("norm1", "q.norm", "k.norm") or name == "final.norm":
            t = 1 + 0.2 * t
        elif base in ("ls1", "ls2"):
            t = 0.7 + 0.2 * t
        elif base == "dwa":
            t = 0.3 * t
            t[-1] += 1
        elif base in ("lq1", "lk1", "lq2", "lk2"):
            t = 0.5 * t * shp[0] ** -0.5
        elif base == "act":
            t = torch.tensor([0.6, -0.4, 0.5, 0.1]) + 0.1 * t
        elif base.startswith("canon"):
            t = 0.5 * t * shp[1] ** -0.5
        elif base.endswith(".b"):
            t = 0.3 * t
        elif base == "router":
            t = 2 * t * shp[-1] ** -0.5
        elif base != "embed":
            t = t * shp[-1] ** -0.5
        out[name] = t.to(torch.bfloat16).to(D)
    return out


def write_model(cfg, sd, folder):
    """The folder layout a user has on disk: config.json and model.safetensors in bfloat16."""
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    head, blobs, off = {}, [], 0
    for name, t in sd.items():
        b = (t.to(torch.bfloat16).view(torch.int16)).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    hb = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hb)) + hb + b"".join(blobs))
