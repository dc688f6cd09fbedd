"""Plain, slow statement of the Luvapel equations: one function per mechanism, whole sequences, no cache, no batch, loops
where a loop is the clearest form.  It shares nothing with the package; the tests compare the two.

Weights are a dict name -> tensor in the checkpoint's own names and [out, in] layout; `cfg` is the plain dict of a
config.json.  Everything is computed in the dtype of the weights (float32 or float64)."""
import math

import torch

from kabadra_oracle import read_safetensors, write_model  # noqa: F401  (test helpers of the other oracle)


def unit_rms(x, eps):
    """Divided by its own root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def unit_length(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


# ---------------------------------------------------------------------------------------------- attention
def rotate_pairs(x, pos, base, dims):
    """x [T, heads, dim]; neighbours (2i, 2i + 1) turn together, the dimensions from `dims` on stay."""
    y = x.clone()
    for i in range(dims // 2):
        ang = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def windowed(q, k, v, scale, size):
    """One head: q [T, d], k [T, d], v [T, e] -> [T, e]; token i sees the `size` tokens up to itself."""
    out = []
    for i in range(q.shape[0]):
        lo = max(0, i - size + 1)
        out.append(torch.softmax(k[lo:i + 1] @ q[i] * scale, 0) @ v[lo:i + 1])
    return torch.stack(out)


def key_value_attention(h, w, m, pre, eps):
    """Windowed attention whose values are the key projections; heads normed one by one, a temperature per head on the
    scores, a gate per output dimension."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    raw_q, raw_k = (h @ w[pre + "q"].T).view(T, H, -1), (h @ w[pre + "k"].T).view(T, G, -1)
    turn = lambda x: rotate_pairs(x, torch.arange(T), m["rot"]["base"], m["rot"]["dims"])
    q, k = turn(unit_rms(raw_q, eps) * w[pre + "q.norm"]), turn(unit_rms(raw_k, eps) * w[pre + "k.norm"])
    out = [windowed(q[:, a], k[:, a // (H // G)], raw_k[:, a // (H // G)], m["scale"] * w[pre + "temp"][a], m["mask"]["size"]) for a in range(H)]
    return (torch.cat(out, 1) * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------- recurrences
def causal_conv(u, w):
    """u [T, channels], w [channels, taps]; the last column belongs to the token itself."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] += w[:, j] * u[t - taps + 1 + j]
    return y


def delta_rule(q, k, v, g, beta, state=None):
    """One head: q, k [T, D], v [T, V], decays g [T], steps beta [T] -> (outputs [T, V], state [D, V])."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype) if state is None else state
    out = []
    for t in range(v.shape[0]):
        S = g[t] * S
        S = S + torch.outer(k[t], beta[t] * (v[t] - S.T @ k[t]))
        out.append(S.T @ q[t])
    return torch.stack(out), S


def gated_delta(h, w, m, pre, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ w[pre + n].T, w[f"{pre}{n}.conv"])) for n in "qkv")
    q, k, v = unit_length(q.view(T, G, D)) * D ** -0.5, unit_length(k.view(T, G, D)), v.view(T, H, V)
    beta = torch.sigmoid(h @ w[pre + "b"].T)
    g = torch.exp(-torch.exp(w[pre + "A_log"]) * softplus(h @ w[pre + "a"].T + w[pre + "dt_bias"]))
    o = torch.stack([delta_rule(q[:, a // (H // G)], k[:, a // (H // G)], v[:, a], g[:, a], beta[:, a])[0] for a in range(H)], 1)
    o = unit_rms(o, eps) * w[pre + "norm"] * silu(h @ w[pre + "g"].T).view(T, H, V)
    return o.reshape(T, -1) @ w[pre + "o"].T


def general_delta_rule(r, k, v, decay, removal, state=None):
    """One head: r, k, v, decay and removal [T, D] -> (outputs [T, D], state [D, D])."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=v.dtype) if state is None else state
    u, out = unit_length(k), []
    for t in range(v.shape[0]):
        S = decay[t][:, None] * S - torch.outer(removal[t] * u[t], S.T @ u[t]) + torch.outer(k[t], v[t])
        out.append(S.T @ r[t])
    return torch.stack(out), S


def general_delta(h, w, m, pre, eps):
    T, H = h.shape[0], m["heads"]
    r, k, v = ((h @ w[pre + n].T).view(T, H, -1) for n in "rkv")
    decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w[pre + "w1"].T) @ w[pre + "w2"].T + w[pre + "w0"])).view(T, H, -1)
    removal = torch.sigmoid(h @ w[pre + "a"].T + w[pre + "a.b"]).view(T, H, -1)
    o = torch.stack([general_delta_rule(r[:, a], k[:, a], v[:, a], decay[:, a], removal[:, a])[0] for a in range(H)], 1)
    return (unit_rms(o, eps).reshape(T, -1) * w[pre + "norm"] * torch.sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def parallel(h, w, m, pre, eps):
    left = key_value_attention(h, w, m["left"], pre + "left.", eps)
    right = gated_delta(h, w, m["right"], pre + "right.", eps)
    return 0.5 * (unit_rms(left, eps) * w[pre + "left.out"] + unit_rms(right, eps) * w[pre + "right.out"])


# ---------------------------------------------------------------------------------------------- layers
def squared_relu_unit(h, w, pre):
    return torch.clamp(h @ w[pre + "up"].T, min=0) ** 2 @ w[pre + "down"].T


def gated_step(x, y, w, gate, norm, eps):
    """The residual after a sublayer that read x and gave y: gated element by element, normed, added."""
    return x + unit_rms(y * torch.sigmoid(x @ w[gate].T + w[gate + ".b"]), eps) * w[norm]


MIXERS = {"parallel": parallel, "general_delta": general_delta}


def forward(cfg, w, tokens, dtype=torch.float32):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        x = gated_step(x, MIXERS[layer["type"]](x, w, layer["mixer"], p + "mix.", eps), w, p + "rg1", p + "norm1", eps)
        if layer["mlp"] is not None:
            x = gated_step(x, squared_relu_unit(x, w, p + "mlp."), w, p + "rg2", p + "norm2", eps)
        stream.append(x)
    return (unit_rms(x, eps) * w["final.norm"]) @ w["head"].T, torch.stack(stream)


# ---------------------------------------------------------------------------------------------- small models for tests
def tensor_shapes(cfg, rank=16):
    """name -> shape of every tensor of a configuration; `rank`: inner size of the decays' two-matrix products."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        if "weights_of" in layer:
            continue
        m, p = layer["mixer"], f"l{i}."
        for n in ("1",) if layer["mlp"] is None else ("1", "2"):
            s[f"{p}norm{n}"], s[f"{p}rg{n}"], s[f"{p}rg{n}.b"] = (W,), (W, W), (W,)
        if layer["mlp"] is not None:
            s[p + "mlp.up"], s[p + "mlp.down"] = (layer["mlp"]["ff"], W), (W, layer["mlp"]["ff"])
        p += "mix."
        if layer["type"] == "general_delta":
            n = m["heads"] * m["dim"]
            for t in "rkvga":
                s[p + t] = (n, W)
            s[p + "a.b"] = s[p + "w0"] = s[p + "norm"] = (n,)
            s[p + "w1"], s[p + "w2"], s[p + "o"] = (rank, W), (n, rank), (W, n)
            continue
        a, q = m["left"], p + "left."
        s[q + "q"], s[q + "k"], s[q + "g"] = (a["heads"] * a["dim"], W), (a["kv_heads"] * a["dim"], W), (a["heads"] * a["vdim"], W)
        s[q + "q.norm"] = s[q + "k.norm"] = (a["dim"],)
        s[q + "temp"], s[q + "o"] = (a["heads"],), (W, a["heads"] * a["vdim"])
        d, q = m["right"], p + "right."
        for t, rows in (("q", d["kv_heads"] * d["dim"]), ("k", d["kv_heads"] * d["dim"]), ("v", d["heads"] * d["vdim"])):
            s[q + t], s[f"{q}{t}.conv"] = (rows, W), (rows, d["conv"])
        s[q + "b"] = s[q + "a"] = (d["heads"], W)
        s[q + "A_log"] = s[q + "dt_bias"] = (d["heads"],)
        s[q + "norm"], s[q + "g"], s[q + "o"] = (d["vdim"],), (d["heads"] * d["vdim"], W), (W, d["heads"] * d["vdim"])
        s[p + "left.out"] = s[p + "right.out"] = (W,)
    return s


def random_weights(cfg, seed=0, rank=16):
    """bfloat16 weights at which every mechanism leaves a mark: scores of a few units, decays between a token and tens of
    tokens, norms and temperatures away from their neutral value, biases."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        t, last = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if "norm" in last or last in ("out", "temp"):
            t = 1.0 + 0.2 * t
        elif last in ("dt_bias", "A_log", "w0", "b") and len(shape) == 1:
            t = 0.5 * t
        elif last != "embed":
            t = t / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
