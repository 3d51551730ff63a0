"""Plain, slow oracle of the Dubazen design: whole sequences, double precision.  One function per mechanism; nothing here is shared with the
product path."""
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


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


# ---------------------------------------------------------------------------------------------- parallel mixer
def rotate(x, base, dims, sign=1):
    """x [T, heads, d]: entries (i, i + dims / 2) of the first ``dims`` turned by sign * position * base^(-2 i / dims)."""
    y, n = x.clone(), dims // 2
    pos = torch.arange(x.shape[0], dtype=x.dtype)[:, None]
    for i in range(n):
        a = sign * pos * base ** (-2.0 * i / dims)
        u, v = x[..., i], x[..., i + n]
        y[..., i], y[..., i + n] = u * torch.cos(a) - v * torch.sin(a), v * torch.cos(a) + u * torch.sin(a)
    return y


def sink_softmax(s, sink):
    """Rows of scores (-inf: not seen) with exp(sink) in the denominator only."""
    m = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def causal(T):
    return torch.tensor([[j <= i for j in range(T)] for i in range(T)])


def attention(h, w, m, eps):
    """Before the output projection: [T, heads * vdim]."""
    H, G, d, e, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    base, dims = m["rot"]["base"], m["rot"]["dims"]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, d)
    k = (h @ w["k"].T + w["k.b"]).reshape(T, G, d)
    v = (h @ w["v"].T + w["v.b"]).reshape(T, G, e)
    q, k = rms(rotate(q, base, dims), eps), rms(rotate(k, base, dims), eps)
    v = rotate(v, base, e)
    o = torch.zeros(T, H, e, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].T * m["scale"]).masked_fill(~causal(T), -math.inf)
        o[:, n] = sink_softmax(s, w["sink"][n]) @ v[:, g]
    return rotate(o, base, e, -1).reshape(T, H * e) * sigmoid(h @ w["g"].T)


def fixed_decay(h, w, m, eps):
    """Linear attention with one constant decay per head."""
    H, d, e, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q, k, v = (silu(h @ w[n].T).reshape(T, H, -1) for n in "qkv")
    S, o = torch.zeros(H, d, e, dtype=h.dtype), torch.zeros(T, H, e, dtype=h.dtype)
    for t in range(T):
        for n in range(H):
            S[n] = m["decay"][n] * S[n] + torch.outer(k[t, n], v[t, n])
            o[t, n] = S[n].T @ q[t, n]
    return (rms(o.reshape(T, H * e), eps) * w["norm"] * sigmoid(h @ w["g"].T)) @ w["o"].T


def parallel(h, w, m, eps):
    a, b = ({k[len(s) + 1:]: t for k, t in w.items() if k.startswith(s + ".")} for s in ("left", "right"))
    left = attention(h, a, m["left"], eps) @ a["o"].T + a["o.b"]
    return m["left_scale"] * left + m["right_scale"] * fixed_decay(h, b, m["right"], eps)


# ---------------------------------------------------------------------------------------------- recurrences
def channel_decay(h, w, m, eps):
    """Gated linear attention: a decay for every key channel."""
    H, d, e, T = m["heads"], m["dim"], m["vdim"], h.shape[0]
    q = (h @ w["q"].T * d ** -0.5).reshape(T, H, d)
    k, v = (h @ w["k"].T).reshape(T, H, d), (h @ w["v"].T).reshape(T, H, e)
    alpha = (sigmoid((h @ w["a1"].T) @ w["a2"].T + w["a2.b"]) ** (1 / m["tau"])).reshape(T, H, d)
    S, o = torch.zeros(H, d, e, dtype=h.dtype), torch.zeros(T, H, e, dtype=h.dtype)
    for t in range(T):
        for n in range(H):
            S[n] = alpha[t, n][:, None] * S[n] + torch.outer(k[t, n], v[t, n])
            o[t, n] = S[n].T @ q[t, n]
    return ((rms(o, eps) * w["norm"]).reshape(T, H * e) * silu(h @ w["g"].T)) @ w["o"].T


def convolution(x, w, b):
    """Per channel, last column the current token, zeros before the sequence."""
    y = b.expand_as(x).clone()
    taps = w.shape[1]
    for t in range(x.shape[0]):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] = y[t] + w[:, j] * x[t - taps + 1 + j]
    return y


def selective_scan(h, w, m, eps):
    I, N, R, T = m["inner"], m["state"], m["dt_rank"], h.shape[0]
    p = h @ w["in"].T
    x, z = silu(convolution(p[:, :I], w["conv"], w["conv.b"])), p[:, I:]
    r = x @ w["x"].T
    dt, B, C = torch.log1p(torch.exp(r[:, :R] @ w["dt"].T + w["dt.b"])), r[:, R:R + N], r[:, R + N:]
    A = -torch.exp(w["A_log"])
    S, y = torch.zeros(I, N, dtype=h.dtype), torch.zeros(T, I, dtype=h.dtype)
    for t in range(T):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t]
        y[t] = S @ C[t] + w["D"] * x[t]
    return (y * silu(z)) @ w["o"].T


MIXERS = {"parallel": parallel, "gla": channel_decay, "mamba1": selective_scan}


# ---------------------------------------------------------------------------------------------- experts
def gated(h, w, name, limit):
    g, u = torch.clamp(h @ w[name + "gate"].T, max=limit), torch.clamp(h @ w[name + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w[name + "down"].T


def route(h, router, top):
    """(experts, weights) of every token: the largest softmax scores over their own sum."""
    z = h @ router.T
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    order = torch.argsort(s, dim=-1, descending=True)[:, :top]
    c = s.gather(1, order)
    return order, c / (c.sum(-1, keepdim=True) + 1e-20)


def mixture(h, w, mlp):
    pick, weight = route(h, w["router"], mlp["router"]["top"])
    y = gated(h, w, "shared.", mlp["shared"]["limit"])
    for t in range(h.shape[0]):
        for e, g in zip(pick[t].tolist(), weight[t]):
            y[t] += g * gated(h[t], w, f"e{e}.", mlp["expert"]["limit"])
    return y


# ---------------------------------------------------------------------------------------------- the stack
def connect(X, p, sub):
    """X [streams, T, W]; p: the sublayer's "in", "out" and "mix" (from, to)."""
    y = sub(torch.einsum("s,stw->tw", p["in"], X))
    return torch.einsum("sr,stw->rtw", p["mix"], X) + p["out"][:, None, None] * y


def forward(cfg, sd, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence (config.json dict, tensors by name)."""
    eps = cfg["norm"]["eps"]
    X = (sd["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]).expand(cfg["streams"], -1, -1)
    for i, lay in enumerate(cfg["layers"]):
        p = f"l{i}."
        sub = {part: {k[len(p) + len(part) + 1:]: t for k, t in sd.items() if k.startswith(p + part + ".")} for part in ("mix", "mlp", "hc1", "hc2")}
        X = connect(X, sub["hc1"], lambda u: MIXERS[lay["type"]](rms(u, eps) * sd[p + "norm1"], sub["mix"], lay["mixer"], eps))
        if lay.get("mlp"):
            X = connect(X, sub["hc2"], lambda u: mixture(rms(u, eps) * sd[p + "norm2"], sub["mlp"], lay["mlp"]))
        if layers_out is not None:
            layers_out.append(X.sum(0))
    return (rms(X.sum(0), eps) * sd["final.norm"]) @ sd["head"].T


# ---------------------------------------------------------------------------------------------- folders
def tensor_shapes(cfg, gla_rank=None):
    """Names and shapes of every tensor of a model folder (the rank of a gla decay stands in no other place than its tensors)."""
    W, out, n = cfg["width"], {}, cfg["streams"]
    out["embed"] = (cfg["vocab"], W)
    for i, lay in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", lay["mixer"], lay.get("mlp")
        q = p + "mix."
        for s in "12" if mlp else "1":
            out.update({f"{p}norm{s}": (), f"{p}hc{s}.in": (n,), f"{p}hc{s}.out": (n,), f"{p}hc{s}.mix": (n, n)})
        if lay["type"] == "parallel":
            a, b = m["left"], m["right"]
            H, G, d, e = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            for t, rows in (("q", H * d), ("k", G * d), ("v", G * e)):
                out[f"{q}left.{t}"], out[f"{q}left.{t}.b"] = (rows, W), (rows,)
            out.update({q + "left.sink": (H,), q + "left.g": (H * e, W), q + "left.o": (W, H * e), q + "left.o.b": (W,)})
            H, d, e = b["heads"], b["dim"], b["vdim"]
            out.update({q + "right.q": (H * d, W), q + "right.k": (H * d, W), q + "right.v": (H * e, W), q + "right.g": (H * e, W),
                        q + "right.o": (W, H * e), q + "right.norm": (H * e,)})
        elif lay["type"] == "gla":
            H, d, e = m["heads"], m["dim"], m["vdim"]
            r = gla_rank or 5
            out.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * e, W), q + "g": (H * e, W), q + "o": (W, H * e), q + "norm": (e,),
                        q + "a1": (r, W), q + "a2": (H * d, r), q + "a2.b": (H * d,)})
        else:
            I, N, R = m["inner"], m["state"], m["dt_rank"]
            out.update({q + "in": (2 * I, W), q + "conv": (I, m["conv"]), q + "conv.b": (I,), q + "x": (R + 2 * N, I), q + "dt": (I, R), q + "dt.b": (I,),
                        q + "A_log": (I, N), q + "D": (I,), q + "o": (W, I)})
        if mlp:
            q, E = p + "mlp.", mlp["router"]["experts"]
            out[q + "router"] = (E, W)
            for name, F in [(f"e{j}", mlp["expert"]["ff"]) for j in range(E)] + [("shared", mlp["shared"]["ff"])]:
                out.update({f"{q}{name}.gate": (F, W), f"{q}{name}.up": (F, W), f"{q}{name}.down": (W, F)})
    out["final.norm"], out["head"] = (), (cfg["vocab"], W)
    return out


def random_model(cfg, seed=0, gla_rank=None):
    """Random bf16-representable weights, spread enough that every one of them matters."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shp in tensor_shapes(cfg, gla_rank).items():
        t = torch.randn(shp, generator=g)
        base = name.split("mix.")[-1] if ".mix." in name else name.split(".")[-1]
        if ".hc" in name:
            n = cfg["streams"]
            t = {"in": 1 / n + 0.3 * t, "out": 1 + 0.3 * t, "mix": 0.7 * torch.eye(n) + 0.3 / n + 0.1 * t}[name.split(".")[-1]]
        elif "norm" in base:
            t = 1 + 0.2 * t
        elif base == "A_log":
            t = torch.log(torch.linspace(0.1, 3.0, shp[1])) + 0.3 * t
        elif base == "dt.b":
            t = -2 + 0.8 * t
        elif base == "a2.b":
            t = 1.5 * t
        elif base == "D":
            t = 1 + 0.3 * t
        elif base == "left.sink":
            t = 1 + t
        elif base == "conv":
            t = t * shp[1] ** -0.5
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
        b = (t.to(torch.bfloat16).contiguous().view(torch.int16)).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [off, off + len(b)]}
        blobs.append(b)
        off += len(b)
    hb = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hb)) + hb + b"".join(blobs))
