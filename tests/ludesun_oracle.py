"""Plain, slow oracle of the Ludesun design: whole sequences, one token at a time where a state is carried, double precision.
One function per mechanism; nothing here is shared with the product path."""
import json
import struct

import numpy as np
import torch

D = torch.float64


def read_safetensors(path):
    raw = open(path, "rb").read()
    n = struct.unpack("<Q", raw[:8])[0]
    head = json.loads(raw[8:8 + n])
    out = {}
    for name, e in head.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        buf = raw[8 + n + a:8 + n + b]
        if e["dtype"] == "BF16":
            t = torch.from_numpy((np.frombuffer(buf, np.uint16).astype(np.uint32) << 16).view(np.float32).copy())
        elif e["dtype"] == "F32":
            t = torch.from_numpy(np.frombuffer(buf, np.float32).copy())
        else:
            t = torch.from_numpy(np.frombuffer(buf, np.int32).copy())
        out[name] = t.reshape(e["shape"]).to(D)
    return out


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh((2 / np.pi) ** 0.5 * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def causal_conv(x, w, b):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    taps = w.shape[1]
    y = torch.zeros_like(x) + b
    for t in range(x.shape[0]):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return y


def mamba2_scan(x, B, C, dt, A_log, Dskip):
    """x [T, H, V], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, V]."""
    T, H, V = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, V, dtype=x.dtype)
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-torch.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + Dskip[h] * x[t, h]
    return y


def grouped_rms(y, groups, eps):
    T, n = y.shape
    return rms(y.reshape(T, groups, n // groups), eps).reshape(T, n)


def mamba2(h, w, m, eps):
    H, V, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, T = H * V, h.shape[0]
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner], xbc[:, inner:inner + G * N], xbc[:, inner + G * N:]
    dt = torch.log1p(torch.exp(-(dt + w["dt_bias"]).abs())) + (dt + w["dt_bias"]).clamp(min=0)
    y = mamba2_scan(x.reshape(T, H, V), B.reshape(T, G, N), C.reshape(T, G, N), dt, w["A_log"], w["D"]).reshape(T, inner)
    return (grouped_rms(y * silu(z), m["norm_groups"], eps) * w["norm"]) @ w["o"].T


def rotate_half(x, pos, base):
    """x [T, ..., dims]: pair (i, i + dims / 2) turned by pos * base^(-2 i / dims)."""
    d = x.shape[-1]
    f = base ** (-2.0 * torch.arange(d // 2, dtype=x.dtype) / d)
    a = (pos.to(x.dtype)[:, None] * f).reshape([x.shape[0]] + [1] * (x.dim() - 2) + [d // 2])
    u, v = x[..., :d // 2], x[..., d // 2:]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin()], -1)


def sink_attention(q, k, v, scale, sink):
    """q / k [T, H, d], v [T, H, e]; exp(sink) joins the denominator."""
    T, H = q.shape[:2]
    o = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T) * scale
        s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), float("-inf"))
        mx = torch.maximum(s.max(-1, keepdim=True).values, sink[h])
        e = torch.exp(s - mx)
        o[:, h] = (e @ v[:, h]) / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - mx))
    return o


def latent_attention(h, w, m, eps):
    H, d, rd, vd, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    pos = torch.arange(T)
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).reshape(T, H, d + rd)
    a = h @ w["dkv"].T
    c = rms(a[:, :r], eps) * w["dkv.norm"]
    kr = rotate_half(a[:, r:].reshape(T, 1, rd), pos, m["rot"]["base"]).expand(T, H, rd)
    q = torch.cat([q[..., :d], rotate_half(q[..., d:], pos, m["rot"]["base"])], -1)
    k = torch.cat([(c @ w["uk"].T).reshape(T, H, d), kr], -1)
    v = (c @ w["uv"].T).reshape(T, H, vd)
    return sink_attention(q, k, v, m["scale"], w["sink"]).reshape(T, H * vd) @ w["o"].T


def mlstm_scan(q, k, v, i, f):
    """q (already scaled) / k [T, H, d], v [T, H, V], log gates i / f [T, H] -> o [T, H, V]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(H, d, dtype=q.dtype)
    m = torch.zeros(H, dtype=q.dtype)
    o = torch.zeros_like(v)
    for t in range(T):
        m2 = torch.maximum(f[t] + m, i[t])
        keep, add = torch.exp(f[t] + m - m2), torch.exp(i[t] - m2)
        m = m2
        for h in range(H):
            S[h] = keep[h] * S[h] + add[h] * torch.outer(k[t, h], v[t, h])
            n[h] = keep[h] * n[h] + add[h] * k[t, h]
            o[t, h] = S[h].T @ q[t, h] / (torch.maximum((n[h] @ q[t, h]).abs(), torch.exp(-m[h])) + 1e-6)
    return o


def mlstm(h, w, m, eps):
    H, d, V, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    T = h.shape[0]
    q = (h @ w["q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w["k"].T).reshape(T, H, d)
    v = (h @ w["v"].T).reshape(T, H, V)
    i = cap * torch.tanh((h @ w["i"].T + w["i.b"]) / cap)
    f = torch.nn.functional.logsigmoid(cap * torch.tanh((h @ w["f"].T + w["f.b"]) / cap))
    o = rms(mlstm_scan(q, k, v, i, f), eps).reshape(T, H * V)
    return (o * w["norm"] * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


MIXERS = {"mamba2": mamba2, "latent_attention": latent_attention, "mlstm": mlstm}


def forward(cfg, sd, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence (config.json dict, tensors by name)."""
    eps = cfg["norm"]["eps"]
    x = sd["embed"][torch.as_tensor(tokens)]
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{lay.get('weights_of', i)}."
        mix = {k[len(p) + 4:]: t for k, t in sd.items() if k.startswith(p + "mix.")}
        x = x + rms(MIXERS[lay["type"]](x, mix, lay["mixer"], eps), eps) * sd[p + "norm1"]
        if lay.get("mlp"):
            y = gelu_tanh(x @ sd[p + "mlp.up"].T) @ sd[p + "mlp.down"].T
            x = x + rms(y, eps) * sd[p + "norm2"]
        if layers_out is not None:
            layers_out.append(x)
    return (rms(x, eps) * sd["final.norm"]) @ sd["head"].T


def tensor_shapes(cfg):
    """Names and shapes of every tensor of a model folder."""
    W, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], W)
    for i, lay in enumerate(cfg["layers"]):
        if "weights_of" in lay:
            continue
        p, m = f"l{i}.", lay["mixer"]
        out[p + "norm1"] = (W,)
        H, V = m["heads"], m["vdim"]
        q = p + "mix."
        if lay["type"] == "mamba2":
            ch = H * V + 2 * m["groups"] * m["state"]
            out.update({q + "in": (H * V + ch + H, W), q + "conv": (ch, m["conv"]), q + "conv.b": (ch,), q + "dt_bias": (H,),
                        q + "A_log": (H,), q + "D": (H,), q + "norm": (H * V,), q + "o": (W, H * V)})
        elif lay["type"] == "latent_attention":
            r, d, rd = m["kv_rank"], m["dim"], m["rot_dim"]
            out.update({q + "dq": (m["q_rank"], W), q + "dq.norm": (m["q_rank"],), q + "uq": (H * (d + rd), m["q_rank"]),
                        q + "dkv": (r + rd, W), q + "dkv.norm": (r,), q + "uk": (H * d, r), q + "uv": (H * V, r), q + "sink": (H,),
                        q + "o": (W, H * V)})
        else:
            d = m["dim"]
            out.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * V, W), q + "g": (H * V, W), q + "o": (W, H * V),
                        q + "norm": (H * V,), q + "i": (H, W), q + "i.b": (H,), q + "f": (H, W), q + "f.b": (H,)})
        if lay.get("mlp"):
            out[p + "norm2"] = (W,)
            out[p + "mlp.up"], out[p + "mlp.down"] = (lay["mlp"]["ff"], W), (W, lay["mlp"]["ff"])
    out["final.norm"], out["head"] = (W,), (cfg["vocab"], W)
    return out


def random_model(cfg, seed=0):
    """Random bf16-representable weights with gates, decays, sinks and norms spread enough to matter."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shp in tensor_shapes(cfg).items():
        t = torch.randn(shp, generator=g)
        base = name.split("mix.")[-1] if "mix." in name else name.split(".")[-1]
        if base in ("norm", "norm1", "norm2", "dq.norm", "dkv.norm"):
            t = 1 + 0.2 * t
        elif base == "A_log":
            t = torch.linspace(-1.5, 1.5, shp[0])
        elif base == "dt_bias":
            t = -1.5 + 0.7 * t
        elif base == "f.b":
            t = 2 + t
        elif base in ("i.b", "sink", "D", "conv.b"):
            t = 0.8 * t
        elif base == "conv":
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
