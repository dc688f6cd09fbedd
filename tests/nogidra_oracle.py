"""Plain, slow statement of the Nogidra equations: one function per mechanism, whole sequences, no cache, no batch, loops
where a loop is the clearest form.  It shares nothing with the package; the tests compare the two.

Weights are a dict name -> tensor in the checkpoint's own names and [out, in] layout; `cfg` is the plain dict of a
config.json.  Everything is computed in the dtype of the weights (float32 or float64)."""
import math

import torch

from kabadra_oracle import read_safetensors, write_model  # noqa: F401  (test helpers of the other oracle)


def unit_rms(x, eps):
    """Divided by its own root mean square."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    """The layers' norm: its weight is stored around zero."""
    return unit_rms(x, eps) * (1 + w)


def linear(h, w, name):
    y = h @ w[name].T
    return y + w[name + ".b"] if name + ".b" in w else y


# ---------------------------------------------------------------------------------------------- positions, windows
def rotate_halves(x, pos, base, dims):
    """x [T, heads, dim]; dimension i < dims/2 turns with dimension i + dims/2, the dimensions from `dims` on stay."""
    y, half = x.clone(), dims // 2
    for i in range(half):
        ang = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i], y[:, :, i + half] = u * c - v * s, v * c + u * s
    return y


def rotate_pairs(x, pos, base, dims):
    """x [T, heads, dim]; neighbours (2i, 2i + 1) turn together."""
    y = x.clone()
    for i in range(dims // 2):
        ang = pos.to(x.dtype) * base ** (-2.0 * i / dims)
        c, s = torch.cos(ang)[:, None], torch.sin(ang)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i], y[:, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return y


def query_temperature(p, coef, every):
    return 1 + coef * math.log((p + 1) // every + 1)


def slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def windowed(q, k, v, scale, size, slope=0.0):
    """One head: q [T, d], k [T, d], v [T, e] -> [T, e]; token i sees the `size` tokens up to itself, and a key at distance
    n costs slope * n."""
    out = []
    for i in range(q.shape[0]):
        lo = max(0, i - size + 1)
        dist = torch.arange(i - lo, -1, -1, dtype=q.dtype)
        s = k[lo:i + 1] @ q[i] * scale - slope * dist
        out.append(torch.softmax(s, 0) @ v[lo:i + 1])
    return torch.stack(out)


def causal_conv(u, w, bias=None):
    """u [T, channels], w [channels, taps]; the last column belongs to the token itself."""
    T, taps = u.shape[0], w.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] += w[:, j] * u[t - taps + 1 + j]
    return y if bias is None else y + bias


# ---------------------------------------------------------------------------------------------- mixers
def attention(h, w, m, pre, eps):
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (causal_conv(h @ w[pre + n].T, w[f"{pre}{n}.conv"]) for n in "qkv")
    q, k, v = q.view(T, H, -1), k.view(T, G, -1), v.view(T, G, -1)
    temp = torch.tensor([query_temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(T)], dtype=h.dtype)
    q = q * temp[:, None, None]
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    out = [windowed(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], m["mask"]["size"], slope(a, H)) * gate[:, a, None]
           for a in range(H)]
    return torch.cat(out, 1) @ w[pre + "o"].T


def latent_attention(h, w, m, pre, eps):
    T, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["kv_rank"], m["vdim"]
    rot = lambda x: rotate_halves(x, torch.arange(T), m["rot"]["base"], m["rot"]["dims"])
    q = (h @ w[pre + "q"].T).view(T, H, D + m["rot_dim"])
    q = torch.cat([q[..., :D], rot(q[..., D:])], -1)
    down = h @ w[pre + "dkv"].T
    c = unit_rms(down[:, :R], eps) * w[pre + "dkv.norm"]
    kr = rot(down[:, None, R:])[:, 0]
    k, v = (c @ w[pre + "uk"].T).view(T, H, D), (c @ w[pre + "uv"].T).view(T, H, V)
    out = [windowed(q[:, a], torch.cat([k[:, a], kr], -1), v[:, a], m["scale"], m["mask"]["size"]) for a in range(H)]
    return torch.cat(out, 1) @ w[pre + "o"].T


def normed_attention(h, w, m, pre, eps):
    """Queries and keys normed over all their heads together, then rotated in neighbouring pairs."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    rot = lambda x: rotate_pairs(x, torch.arange(T), m["rot"]["base"], m["rot"]["dims"])
    q = rot((unit_rms(linear(h, w, pre + "q"), eps) * w[pre + "q.norm"]).view(T, H, -1))
    k = rot((unit_rms(linear(h, w, pre + "k"), eps) * w[pre + "k.norm"]).view(T, G, -1))
    v = linear(h, w, pre + "v").view(T, G, -1)
    out = [windowed(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], m["mask"]["size"]) for a in range(H)]
    return torch.cat(out, 1) @ w[pre + "o"].T


def state_space(x, B, C, dt, A_log, D, state=None):
    """One head: x [T, V], B, C [T, N], dt [T] -> (y [T, V], state [N, V])."""
    S = torch.zeros(B.shape[1], x.shape[1], dtype=x.dtype) if state is None else state
    y = []
    for t in range(x.shape[0]):
        S = torch.exp(-torch.exp(A_log) * dt[t]) * S + dt[t] * torch.outer(B[t], x[t])
        y.append(S.T @ C[t] + D * x[t])
    return torch.stack(y), S


def group_norm(y, w, groups, eps):
    T = y.shape[0]
    return unit_rms(y.view(T, groups, -1), eps).reshape(T, -1) * w


def mamba2(h, w, m, pre, eps):
    T, H, V, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * V
    z, xbc, dt = (h @ w[pre + "in"].T).split([inner, inner + 2 * G * N, H], 1)
    xbc = torch.nn.functional.silu(causal_conv(xbc, w[pre + "conv"], w[pre + "conv.b"]))
    x, B, C = xbc.split([inner, G * N, G * N], 1)
    x, B, C = x.view(T, H, V), B.view(T, G, N), C.view(T, G, N)
    dt = torch.nn.functional.softplus(dt + w[pre + "dt_bias"], threshold=1e9)
    y = [state_space(x[:, a], B[:, a // (H // G)], C[:, a // (H // G)], dt[:, a], w[pre + "A_log"][a], w[pre + "D"][a])[0] for a in range(H)]
    y = torch.cat(y, 1) * torch.nn.functional.silu(z)
    return group_norm(y, w[pre + "norm"], m["norm_groups"], eps) @ w[pre + "o"].T


def parallel(h, w, m, pre, eps):
    return (m["left_scale"] * normed_attention(h, w, m["left"], pre + "left.", eps)
            + m["right_scale"] * mamba2(h, w, m["right"], pre + "right.", eps))


# ---------------------------------------------------------------------------------------------- feed-forward
def gated_unit(h, w, pre):
    g = linear(h, w, pre + "gate")
    return linear(g * torch.sigmoid(g) * linear(h, w, pre + "up"), w, pre + "down")


def route(h, w_router, top):
    """(chosen experts [T, top], their weights [T, top]) of every token."""
    z, ids = (h @ w_router.T).topk(top, -1)
    return ids, torch.softmax(z, -1)


def experts(h, w, f, pre):
    ids, weights = route(h, w[pre + "router"], f["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), weights[t]):
            out[t] += a * gated_unit(h[t], w, f"{pre}e{e}.")
    return out


def feed_forward(h, w, f, pre):
    return gated_unit(h, w, pre) if f["kind"] == "dense" else experts(h, w, f, pre)


# ---------------------------------------------------------------------------------------------- model
MIXERS = {"attention": attention, "latent_attention": latent_attention, "parallel": parallel}


def forward(cfg, w, tokens, dtype=torch.float32):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](norm(x, w[p + "norm1"], eps), w, layer["mixer"], p + "mix.", eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(norm(x, w[p + "norm2"], eps), w, layer["mlp"], p + "mlp.")
        stream.append(x)
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(norm(x, w["final.norm"], eps) @ w["head"].T / cap), torch.stack(stream)


# ---------------------------------------------------------------------------------------------- small models for tests
def tensor_shapes(cfg):
    """name -> shape of every tensor of a configuration."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        m, f, p = layer["mixer"], layer["mlp"], f"l{i}."
        s[p + "norm1"] = (W,)
        if f is not None:
            s[p + "norm2"] = (W,)
            ff = f["ff"] if f["kind"] == "dense" else f["expert"]["ff"]
            units = [""] if f["kind"] == "dense" else [f"e{e}." for e in range(f["router"]["experts"])]
            for u in units:
                for n, shape in (("gate", (ff, W)), ("up", (ff, W)), ("down", (W, ff))):
                    s[f"{p}mlp.{u}{n}"] = shape
                    if u == "":
                        s[f"{p}mlp.{n}.b"] = shape[:1]
            if f["kind"] == "moe":
                s[p + "mlp.router"] = (f["router"]["experts"], W)
        p += "mix."
        if layer["type"] == "latent_attention":
            H, D, R, P, E = m["heads"], m["dim"], m["kv_rank"], m["rot_dim"], m["vdim"]
            s[p + "q"], s[p + "dkv"], s[p + "dkv.norm"] = (H * (D + P), W), (R + P, W), (R,)
            s[p + "uk"], s[p + "uv"], s[p + "o"] = (H * D, R), (H * E, R), (W, H * E)
            continue
        a, q = (m["left"], p + "left.") if layer["type"] == "parallel" else (m, p)
        for n, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
            s[q + n] = (rows, W)
            if layer["type"] == "attention":
                s[f"{q}{n}.conv"] = (rows, m["conv"])
            else:
                s[f"{q}{n}.b"] = (rows,)
                if n != "v":
                    s[f"{q}{n}.norm"] = (rows,)
        s[q + "o"] = (W, a["heads"] * a["vdim"])
        if layer["type"] == "attention":
            s[p + "g"] = (m["heads"], W)
            continue
        r, q = m["right"], p + "right."
        inner, bc = r["heads"] * r["vdim"], r["groups"] * r["state"]
        s[q + "in"], s[q + "o"], s[q + "norm"] = (2 * inner + 2 * bc + r["heads"], W), (W, inner), (inner,)
        s[q + "conv"], s[q + "conv.b"] = (inner + 2 * bc, r["conv"]), (inner + 2 * bc,)
        s[q + "dt_bias"] = s[q + "A_log"] = s[q + "D"] = (r["heads"],)
    return s


def random_weights(cfg, seed=0, decisive=False):
    """bfloat16 weights at which every mechanism leaves a mark: scores of a few units, decays between a token and tens of
    tokens, norms away from their neutral value, biases.  `decisive`: one channel of the residual is a constant that no layer
    touches, and the routers see it with weights so far apart that every token chooses the same experts, whatever the
    precision of its scores."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t, last = torch.randn(shape, generator=g), name.rsplit(".", 1)[-1]
        if "norm" in last:
            t = (1.0 if ".mix." in name else 0.0) + 0.2 * t
        elif last == "b" or last in ("dt_bias", "A_log"):
            t = 0.4 * t
        elif last not in ("embed", "D"):
            t = t * (1.7 if last == "router" else 1.0) / math.sqrt(shape[-1])
        if decisive:
            if name == "embed":
                t[:, 0] = 4.0
            elif last in ("o", "down") or name.endswith("down.b"):
                t[0] = 0.0
            elif last == "router":
                t = 0.1 * t
                t[:, 0] = 1.5 * torch.randperm(shape[0], generator=g)
            elif name.endswith("norm2"):
                t[0] = 0.0
        out[name] = t.to(torch.bfloat16)
    return out
