"""Plain, slow statement of the Kabadra equations: one function per mechanism, whole sequences, no cache, no batch,
loops where a loop is the clearest form.  It shares nothing with the package; the tests compare the two.

Weights are a dict name -> tensor in the checkpoint's own names and [out, in] layout; `cfg` is the plain dict of a
config.json.  Everything is computed in the dtype of the weights (float32 or float64)."""
import json
import math
import struct

import torch


def read_safetensors(path):
    """name -> tensor of a safetensors file: 8-byte length, JSON header, raw data."""
    kinds = {"BF16": torch.bfloat16, "F32": torch.float32, "F16": torch.float16, "I32": torch.int32}
    with open(path, "rb") as f:
        n = struct.unpack("<Q", f.read(8))[0]
        head = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, d in head.items():
        if name == "__metadata__":
            continue
        a, b = d["data_offsets"]
        out[name] = torch.frombuffer(bytearray(data[a:b]), dtype=kinds[d["dtype"]]).reshape(d["shape"])
    return out


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def embedding(tokens, embed, pos, norm_w, eps):
    """Token vector + learned vector of the position, then a norm."""
    rows = [embed[t] + pos[p] for p, t in enumerate(tokens)]
    return rms_norm(torch.stack(rows), norm_w, eps)


def latent(h, w_dkv, norm_w, eps):
    return rms_norm(h @ w_dkv.T, norm_w, eps)


def window_keys(i, size):
    """Positions that position i attends to."""
    return list(range(max(0, i - size + 1), i + 1))


def sink_softmax(scores, sink):
    """Weights over the keys when exp(sink) is part of the denominator."""
    m = max(float(scores.max()), float(sink))
    e = torch.exp(scores - m)
    return e / (e.sum() + torch.exp(sink - m))


def latent_attention(h, c, w, m, pre):
    """h [T, width], c [T, kv_rank]; w the weights, m the mixer's sizes, pre the tensors' prefix."""
    T, H, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).view(T, H, dim)
    k = (c @ w[pre + "uk"].T).view(T, H, dim)
    v = (c @ w[pre + "uv"].T).view(T, H, vdim)
    gate = torch.sigmoid(h @ w[pre + "g"].T)
    out = torch.zeros(T, H, vdim, dtype=h.dtype)
    for i in range(T):
        js = window_keys(i, m["mask"]["size"])
        for a in range(H):
            s = (k[js, a] @ q[i, a]) * m["scale"]
            out[i, a] = sink_softmax(s, w[pre + "sink"][a]) @ v[js, a] * gate[i, a]
    return out.reshape(T, H * vdim) @ w[pre + "o"].T


def clamped_glu(h, w_gate, w_up, w_down, limit):
    g = torch.minimum(h @ w_gate.T, torch.tensor(limit, dtype=h.dtype))
    u = torch.clamp(h @ w_up.T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w_down.T


def forward(cfg, w, tokens, dtype=torch.float32):
    """(logits [T, vocab], residual stream after every layer [layers, T, width])."""
    w = {k: v.to(dtype) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = embedding(tokens, w["embed"], w["pos"], w["embed.norm"], eps)
    latents, stream = {}, []
    for i, layer in enumerate(cfg["layers"]):
        h = rms_norm(x, w[f"l{i}.norm1"], eps)
        m, pre = layer["mixer"], f"l{i}.mix."
        src = m.get("kv_from")
        if src is None:
            latents[i] = latent(h, w[pre + "dkv"], w[pre + "dkv.norm"], eps)
        y = latent_attention(h, latents[i if src is None else src], w, m, pre)
        if layer["mlp"] is not None:
            p = f"l{i}.mlp."
            y = y + clamped_glu(h, w[p + "gate"], w[p + "up"], w[p + "down"], layer["mlp"]["limit"])
        x = x + y
        stream.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg["logit_scale"], torch.stack(stream)


# ---------------------------------------------------------------------------------------------- small models for tests
def tensor_shapes(cfg):
    """name -> shape of every tensor of a configuration."""
    W, V = cfg["width"], cfg["vocab"]
    s = {"embed": (V, W), "pos": (cfg["max_positions"], W), "embed.norm": (W,), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        H, R = m["heads"], m["kv_rank"]
        s[p + "norm1"] = (W,)
        s[p + "mix.q"] = (H * m["dim"], W)
        if m.get("kv_from") is None:
            s[p + "mix.dkv"] = (R, W)
            s[p + "mix.dkv.norm"] = (R,)
        s[p + "mix.uk"] = (H * m["dim"], R)
        s[p + "mix.uv"] = (H * m["vdim"], R)
        s[p + "mix.sink"] = (H,)
        s[p + "mix.g"] = (H, W)
        s[p + "mix.o"] = (W, H * m["vdim"])
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            s[p + "mlp.gate"], s[p + "mlp.up"], s[p + "mlp.down"] = (f, W), (f, W), (W, f)
    return s


def random_weights(cfg, seed=0, gain=1.0):
    """bfloat16 weights at which every mechanism leaves a mark: unit-scale products, norms away from 1, sinks of the
    size of the scores."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if name.endswith("norm") or name.endswith("norm1"):
            t = 1.0 + 0.2 * t
        elif name.endswith(".sink"):
            t = 1.5 * t
        elif name in ("embed", "pos"):
            t = t * 0.7
        elif name.endswith((".uk", ".q")):
            t = t * gain * 1.3 / math.sqrt(shape[-1])
        else:
            t = t * gain / math.sqrt(shape[-1])
        out[name] = t.to(torch.bfloat16)
    return out


def write_model(folder, cfg, weights):
    """config.json and model.safetensors of a small model."""
    import os
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    head, blobs, at = {}, [], 0
    for name, t in weights.items():
        b = t.contiguous().view(torch.int16).numpy().tobytes()
        head[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [at, at + len(b)]}
        blobs.append(b)
        at += len(b)
    h = json.dumps(head).encode()
    h += b" " * (-len(h) % 8)
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h + b"".join(blobs))
    return folder
