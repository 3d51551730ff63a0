"""Plain, slow oracle of the Lanilix design: whole sequences, one token at a time where a state is carried, double precision.
One function per mechanism; nothing here is shared with the product path."""
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


def norm(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def softplus(z):
    return z.clamp(min=0) + torch.log1p(torch.exp(-z.abs()))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def short_conv(x, w):
    """silu of a causal convolution per channel: x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    taps = w.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return silu(y)


def delta_scan(q, k, v, beta, decay):
    """Gated delta rule: q / k [T, G, d] (unit vectors, q scaled), v [T, H, e], beta / decay [T, H] -> (o [T, H, e], S [H, d, e])."""
    T, H, e = v.shape
    G, d = q.shape[1:]
    S = torch.zeros(H, d, e, dtype=v.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // (H // G)], q[t, h // (H // G)]
            s = decay[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - s.T @ kk)
            S[h] = s + torch.outer(kk, u)
            o[t, h] = S[h].T @ qq
    return o, S


def delta(h, w, m, eps):
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    q = unit(short_conv(h @ w["q"].T, w["q.conv"]).reshape(T, G, d)) * d ** -0.5
    k = unit(short_conv(h @ w["k"].T, w["k.conv"]).reshape(T, G, d))
    v = short_conv(h @ w["v"].T, w["v.conv"]).reshape(T, H, e)
    beta = 1 / (1 + torch.exp(-(h @ w["b"].T)))
    decay = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o, _ = delta_scan(q, k, v, beta, decay)
    return ((rms(o, eps) * w["norm"]).reshape(T, H * e) * silu(h @ w["g"].T)) @ w["o"].T


def rotate_pairs(x, pos, base, dims):
    """x [T, heads, d]: neighbours (2 i, 2 i + 1) of the first ``dims`` entries turned by pos * base^(-2 i / dims)."""
    y = x.clone()
    for i in range(dims // 2):
        a = pos.to(x.dtype)[:, None] * base ** (-2.0 * i / dims)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * a.cos() - v * a.sin()
        y[..., 2 * i + 1] = v * a.cos() + u * a.sin()
    return y


def visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def window_attention(q, k, v, scale, size, keep_first):
    """q [T, H, d], k [T, G, d], v [T, G, e]: softmax over the keys of a sliding window and the first tokens of the sequence."""
    T, H = q.shape[:2]
    G = k.shape[1]
    seen = torch.tensor([[visible(i, j, size, keep_first) for j in range(T)] for i in range(T)])
    o = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        o[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, h // (H // G)]
    return o


def attention(h, w, m, eps):
    H, G, d, T = m["heads"], m["kv_heads"], m["dim"], h.shape[0]
    assert m["vdim"] == d
    pos = torch.arange(T)
    kp = h @ w["k"].T
    q = (rms(h @ w["q"].T, eps) * w["q.norm"]).reshape(T, H, d)
    k = (rms(kp, eps) * w["k.norm"]).reshape(T, G, d)
    q, k = (rotate_pairs(t, pos, m["rot"]["base"], m["rot"]["dims"]) for t in (q, k))
    o = window_attention(q, k, kp.reshape(T, G, d), m["scale"], m["mask"]["size"], m["mask"]["keep_first"])
    return o.reshape(T, H * d) @ w["o"].T


def clamped_glu(x, w_gate, w_up, w_down, limit):
    g = (x @ w_gate.T).clamp(max=limit)
    u = (x @ w_up.T).clamp(-limit, limit)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ w_down.T


MIXERS = {"delta": delta, "attention": attention}


def forward(cfg, sd, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence (config.json dict, tensors by name)."""
    eps = cfg["norm"]["eps"]
    x = sd["embed"][torch.as_tensor(tokens)]
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{lay.get('weights_of', i)}."
        mix = {k[len(p) + 4:]: t for k, t in sd.items() if k.startswith(p + "mix.")}
        x = x + norm(MIXERS[lay["type"]](norm(x, sd[p + "norm1"], eps), mix, lay["mixer"], eps), sd[p + "norm1b"], eps)
        if lay.get("mlp"):
            y = clamped_glu(norm(x, sd[p + "norm2"], eps), sd[p + "mlp.gate"], sd[p + "mlp.up"], sd[p + "mlp.down"], lay["mlp"]["limit"])
            x = x + norm(y, sd[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return norm(x, sd["final.norm"], eps) @ sd["head"].T


def tensor_shapes(cfg):
    """Names and shapes of every tensor of a model folder."""
    W, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], W)
    for i, lay in enumerate(cfg["layers"]):
        if "weights_of" in lay:
            continue
        p, m = f"l{i}.", lay["mixer"]
        q = p + "mix."
        out[p + "norm1"] = out[p + "norm1b"] = (W,)
        H, G, d, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        if lay["type"] == "delta":
            for n, ch in (("q", G * d), ("k", G * d), ("v", H * V)):
                out[q + n], out[q + n + ".conv"] = (ch, W), (ch, m["conv"])
            out.update({q + "a": (H, W), q + "b": (H, W), q + "A_log": (H,), q + "dt_bias": (H,), q + "norm": (V,), q + "g": (H * V, W), q + "o": (W, H * V)})
        else:
            out.update({q + "q": (H * d, W), q + "k": (G * d, W), q + "q.norm": (H * d,), q + "k.norm": (G * d,), q + "o": (W, H * V)})
        if lay.get("mlp"):
            F = lay["mlp"]["ff"]
            out[p + "norm2"] = out[p + "norm2b"] = (W,)
            out.update({p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    out["final.norm"], out["head"] = (W,), (cfg["vocab"], W)
    return out


def random_model(cfg, seed=0):
    """Random bf16-representable weights with gates, decays and norms spread enough to matter."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shp in tensor_shapes(cfg).items():
        t = torch.randn(shp, generator=g)
        base = name.split("mix.")[-1] if "mix." in name else name.split(".")[-1]
        if base in ("norm1", "norm1b", "norm2", "norm2b") or name == "final.norm":
            t = 0.2 * t
        elif base in ("norm", "q.norm", "k.norm"):
            t = 1 + 0.2 * t
        elif base == "A_log":
            t = torch.linspace(-2.5, 1.0, shp[0])
        elif base == "dt_bias":
            t = -1.5 + 0.7 * t
        elif base.endswith(".conv"):
            t = t * shp[1] ** -0.5
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
