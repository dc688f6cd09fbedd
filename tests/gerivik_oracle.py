"""Plain, slow statement of the Gerivik equations: one function per mechanism, whole sequences, no cache, no batch, loops
where a loop is the clearest form.  It shares nothing with the package; the tests compare the two.

Weights are a dict name -> tensor in the checkpoint's own names and [out, in] layout; `cfg` is the plain dict of a
config.json.  Everything is computed in the dtype of the weights (float32 or float64)."""
import math

import torch

from kabadra_oracle import read_safetensors, rms_norm, write_model  # noqa: F401  (test helpers of the other oracle)


# ---------------------------------------------------------------------------------------------- attention
def unit_rms(x, eps):
    """Divided by its own root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate(x, pos, base, dims):
    """x [T, heads, dim]; dimension i < dims/2 turns with dimension i + dims/2, the dimensions from `dims` on stay."""
    y, half = x.clone(), dims // 2
    for i in range(half):
        ang = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i], y[:, :, i + half] = u * c - v * s, v * c + u * s
    return y


def capped(score, cap):
    return cap * torch.tanh(score / cap)


def attention(h, w, m, pre, eps):
    """Causal softmax attention with capped scores; h [T, width]."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[pre + "q"].T).view(T, H, m["dim"])
    k = (h @ w[pre + "k"].T).view(T, G, m["dim"])
    v = (h @ w[pre + "v"].T).view(T, G, m["vdim"])
    pos = torch.arange(T)
    q = unit_rms(rotate(q, pos, m["rot"]["base"], m["rot"]["dims"]), eps)
    k = unit_rms(rotate(k, pos, m["rot"]["base"], m["rot"]["dims"]), eps)
    out = torch.zeros(T, H, m["vdim"], dtype=h.dtype)
    for i in range(T):
        for a in range(H):
            g = a // (H // G)
            s = capped(k[:i + 1, g] @ q[i, a] * m["scale"], m["softcap"])
            out[i, a] = torch.softmax(s, 0) @ v[:i + 1, g]
    return out.reshape(T, -1) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------- gated linear attention
def channel_decay(h, w_a1, w_a2, bias, tau):
    """Factor in (0, 1) per token and key channel."""
    return torch.sigmoid((h @ w_a1.T) @ w_a2.T + bias) ** (1.0 / tau)


def recurrence(q, k, v, alpha, state=None):
    """q, k, alpha [T, dim], v [T, vdim] of one head: (outputs [T, vdim], state [dim, vdim])."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        S = alpha[t][:, None] * S + torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def gla(h, w, m, pre, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, D) * D ** -0.5
    k = (h @ w[pre + "k"].T).view(T, H, D)
    v = (h @ w[pre + "v"].T).view(T, H, V)
    alpha = channel_decay(h, w[pre + "a1"], w[pre + "a2"], w[pre + "a2.b"], m["tau"]).view(T, H, D)
    o = torch.stack([recurrence(q[:, a], k[:, a], v[:, a], alpha[:, a])[0] for a in range(H)], 1)
    o = rms_norm(o, w[pre + "norm"], eps).reshape(T, H * V)
    return (o * torch.nn.functional.silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---------------------------------------------------------------------------------------------- experts
def route(h, w_router, correction, r):
    """(chosen experts [T, top], their weights [T, top]) of every token."""
    n = r["experts"] + r["identity"]
    s = torch.softmax(h @ w_router.T, -1)
    size = n // r["groups"]["count"]
    ids, weights = [], []
    for t in range(h.shape[0]):
        choice = s[t] + correction
        best = torch.stack([choice[g * size:(g + 1) * size].max() for g in range(r["groups"]["count"])])
        kept = set(best.topk(r["groups"]["keep"]).indices.tolist())
        choice = torch.stack([choice[e] if e // size in kept else torch.tensor(-math.inf, dtype=s.dtype) for e in range(n)])
        top = choice.topk(r["top"]).indices
        ids.append(top)
        weights.append(s[t][top])
    return torch.stack(ids), torch.stack(weights)


def expert(h, w_gate, w_up, w_down, limit):
    g = torch.minimum(h @ w_gate.T, torch.tensor(limit, dtype=h.dtype))
    u = torch.clamp(h @ w_up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w_down.T


def experts(h, w, f, pre):
    ids, weights = route(h, w[pre + "router"], w[pre + "correction"], f["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), weights[t]):
            if e >= f["router"]["experts"]:
                y = h[t]
            else:
                p = f"{pre}e{e}."
                y = expert(h[t], w[p + "gate"], w[p + "up"], w[p + "down"], f["expert"]["limit"])
            out[t] += a * y
    return out


# ---------------------------------------------------------------------------------------------- model
def forward(cfg, w, tokens, dtype=torch.float32):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{layer.get('weights_of', i)}."
        mixer = {"attention": attention, "gla": gla}[layer["type"]]
        x = x + rms_norm(mixer(rms_norm(x, w[p + "norm1"], eps), w, layer["mixer"], p + "mix.", eps), w[p + "norm1b"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(experts(rms_norm(x, w[p + "norm2"], eps), w, layer["mlp"], p + "mlp."), w[p + "norm2b"], eps)
        stream.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T, torch.stack(stream)


# ---------------------------------------------------------------------------------------------- small models for tests
def tensor_shapes(cfg, rank=None):
    """name -> shape of every tensor of a configuration; `rank`: rows of the decay's first matrix, by layer (default 8)."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        H, D, E = m["heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f is not None else ()):
            s[p + n] = (W,)
        p += "mix."
        s[p + "q"], s[p + "o"] = (H * D, W), (W, H * E)
        if layer["type"] == "attention":
            s[p + "k"], s[p + "v"] = (m["kv_heads"] * D, W), (m["kv_heads"] * E, W)
        else:
            r = 8 if rank is None else rank[i]
            s[p + "k"], s[p + "v"], s[p + "g"], s[p + "norm"] = (H * D, W), (H * E, W), (H * E, W), (E,)
            s[p + "a1"], s[p + "a2"], s[p + "a2.b"] = (r, W), (H * D, r), (H * D,)
        if f is not None:
            p = f"l{i}.mlp."
            n = f["router"]["experts"]
            s[p + "router"], s[p + "correction"] = (n + f["router"]["identity"], W), (n + f["router"]["identity"],)
            for e in range(n):
                s[f"{p}e{e}.gate"] = s[f"{p}e{e}.up"] = (f["expert"]["ff"], W)
                s[f"{p}e{e}.down"] = (W, f["expert"]["ff"])
    return s


def random_weights(cfg, seed=0, rank=None):
    """bfloat16 weights at which every mechanism leaves a mark: scores of a few units, decays between a token and a
    hundred tokens, router scores and corrections of like size, norms away from 1."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        t = torch.randn(shape, generator=g)
        if "norm" in name.rsplit(".", 1)[-1]:
            t = 1.0 + 0.2 * t
        elif name == "embed":
            t = t * 0.3
        elif name.endswith(".correction"):
            t = 0.15 * t
        elif name.endswith(".a2.b"):
            t = 1.5 * t
        elif name.endswith(".router"):
            t = 1.7 * t / math.sqrt(shape[-1])
        else:
            t = t / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out
