"""Plain, slow implementation of the Folirax design, one function per mechanism, for comparison with the framework.

Written from the equations alone: torch tensors on the CPU, in the dtype the caller picks (float64 or float32), one sequence at
a time, and nothing imported from the package.  ``W`` is a dict of tensors by their names in a checkpoint.
"""
import json
import math
import os
import struct

import numpy as np
import torch


# ---------------------------------------------------------------- checkpoints
def write_safetensors(path, tensors):
    """The container: header length, JSON header, raw little-endian data (bf16 for floats)."""
    header, blobs, off = {}, [], 0
    for name, t in tensors.items():
        t = t.detach().contiguous()
        if t.is_floating_point():
            raw, dt = t.to(torch.bfloat16).view(torch.int16).numpy().tobytes(), "BF16"
        else:
            raw, dt = t.to(torch.int32).numpy().tobytes(), "I32"
        header[name] = {"dtype": dt, "shape": list(t.shape), "data_offsets": [off, off + len(raw)]}
        blobs.append(raw)
        off += len(raw)
    h = json.dumps(header).encode()
    h += b" " * (-len(h) % 8)
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(h)) + h)
        for b in blobs:
            f.write(b)


def read_safetensors(path):
    data = open(path, "rb").read()
    n = struct.unpack("<Q", data[:8])[0]
    header = json.loads(data[8: 8 + n])
    out = {}
    for name, e in header.items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        raw = data[8 + n + a: 8 + n + b]
        if e["dtype"] == "BF16":
            x = torch.from_numpy(np.frombuffer(raw, dtype="<i2").copy()).view(torch.bfloat16)
        else:
            x = torch.from_numpy(np.frombuffer(raw, dtype={"I32": "<i4", "F32": "<f4"}[e["dtype"]]).copy())
        out[name] = x.reshape(e["shape"])
    return out


def load(folder, dtype=torch.float64):
    cfg = json.load(open(os.path.join(folder, "config.json")))
    W = read_safetensors(os.path.join(folder, "model.safetensors"))
    return cfg, {k: v.to(dtype) if v.is_floating_point() else v for k, v in W.items()}


# ---------------------------------------------------------------- mechanisms
def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1 + w)


def rotate(x, pos, dims, base):
    """x [T, heads, dim]: the first ``dims`` dimensions of every head turn in adjacent pairs, pair i by pos * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = (pos.to(torch.float64) * base ** (-2.0 * i / dims)).to(x.dtype)[:, None]
        c, s = torch.cos(a), torch.sin(a)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def softmax_attention(q, k, v, scale, first_pos):
    """q [T, H, dim] at positions first_pos..; k [S, G, dim], v [S, G, vdim] from position 0: causal, ordinary softmax."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    k, v = k.repeat_interleave(H // G, 1), v.repeat_interleave(H // G, 1)
    s = torch.einsum("thd,shd->hts", q, k) * scale
    visible = torch.arange(S)[None, :] <= (first_pos + torch.arange(T))[:, None]
    s = s.masked_fill(~visible[None], -math.inf)
    return torch.einsum("hts,shv->thv", torch.softmax(s, -1), v)


def attention_mixer(h, W, p, mx, eps, pos0, cache, owner):
    """One attention mixer on rows h [T, width]; ``cache[layer]`` = (keys, values) as stored; ``owner`` = whose cache it reads."""
    T = h.shape[0]
    H, G, dim, vdim = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    pos = torch.arange(pos0, pos0 + T)
    rot = mx["rot"]
    q = rms(rotate((h @ W[p + "q"].T).view(T, H, dim), pos, rot["dims"], rot["base"]), eps)
    if mx.get("kv_from") is None:
        k = rms(rotate((h @ W[p + "k"].T).view(T, G, dim), pos, rot["dims"], rot["base"]), eps)
        v = (h @ W[p + "v"].T).view(T, G, vdim)
        old = cache.get(owner)
        cache[owner] = (k, v) if old is None else (torch.cat([old[0], k]), torch.cat([old[1], v]))
    ks, vs = cache[owner]
    o = softmax_attention(q, ks, vs, mx["scale"], pos0)
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * vdim) @ W[p + "o"].T


def log_decay(h, W, p, tau):
    """log of the per-channel decay: log sigmoid(z) / tau with z = A2 (A1 h) + b."""
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    return torch.nn.functional.logsigmoid(z) / tau


def gla_recurrence(q, k, v, g, S):
    """Token by token: S [H, dim, vdim] decays per key channel, takes k v^T, and is read by q.  q, k, g [T, H, dim]; v [T, H, vdim]."""
    out = []
    for t in range(q.shape[0]):
        S = torch.exp(g[t])[..., None] * S + k[t][..., None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gla_mixer(h, W, p, mx, eps, layer, state):
    T = h.shape[0]
    H, dim, vdim = mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, dim) * dim ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, dim)
    v = (h @ W[p + "v"].T).view(T, H, vdim)
    g = log_decay(h, W, p, mx["tau"]).view(T, H, dim)
    S = state.get(layer)
    if S is None:
        S = torch.zeros(H, dim, vdim, dtype=h.dtype)
    o, state[layer] = gla_recurrence(q, k, v, g, S)
    o = (rms(o, eps) * W[p + "norm"]).reshape(T, H * vdim)
    o = o * torch.nn.functional.silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T


def relu2_ff(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def finish_logits(x, W, cfg):
    y = centred_norm(x, W["final.norm"], cfg["norm"]["eps"]) @ W["head"].T * cfg["logit_scale"]
    c = cfg["logit_softcap"]
    return c * torch.tanh(y / c)


class Sequence:
    """What one sequence has left behind: keys and values per attention layer that owns some, state per recurrent layer."""

    def __init__(self):
        self.cache, self.state, self.length = {}, {}, 0


def forward(cfg, W, tokens, seq, layers_out=None):
    """Append ``tokens``; logits [T, vocab] of every one.  ``layers_out``: a list that takes the residual after every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        h = centred_norm(x, W[p + "norm1"], eps)
        if L["type"] == "gla":
            y = gla_mixer(h, W, p + "mix.", mx, eps, i, seq.state)
        else:
            owner = i if mx.get("kv_from") is None else mx["kv_from"]
            y = attention_mixer(h, W, p + "mix.", mx, eps, seq.length, seq.cache, owner)
        x = x + centred_norm(y, W[p + "norm1b"], eps)
        if L.get("mlp") is not None:
            y = relu2_ff(centred_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
            x = x + centred_norm(y, W[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    seq.length += len(tokens)
    return finish_logits(x, W, cfg)


def generate(cfg, W, prompt, n):
    """Greedy continuation; returns the ids and the logits each was taken from."""
    seq = Sequence()
    row = forward(cfg, W, prompt, seq)[-1]
    ids, rows = [], []
    for _ in range(n):
        ids.append(int(row.argmax()))
        rows.append(row)
        row = forward(cfg, W, [ids[-1]], seq)[-1]
    return ids, torch.stack(rows)


# ---------------------------------------------------------------- small random models
def layer_attention(dim, vdim, heads, kv_heads, rot_dims, base=10000.0, scale=None, ff=None, kv_from=None):
    mx = {"dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv_heads, "rot": {"base": base, "dims": rot_dims},
          "scale": dim ** -0.5 if scale is None else scale}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "attention", "mixer": mx, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def layer_gla(dim, vdim, heads, tau=16.0, ff=None):
    return {"type": "gla", "mixer": {"dim": dim, "vdim": vdim, "heads": heads, "tau": tau},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, eps=1e-6, logit_scale=0.7, softcap=20.0):
    return {"architecture": "Folirax", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps},
            "logit_scale": logit_scale, "logit_softcap": softcap}


def random_weights(cfg, seed=0, rank=8):
    """Seeded weights, rounded to bf16 (what a checkpoint holds), returned in float64."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def put(name, *shape, std=None, mean=0.0):
        s = shape[-1] ** -0.5 if std is None else std
        W[name] = (torch.randn(*shape, generator=g, dtype=torch.float64) * s + mean).to(torch.bfloat16).double()

    d = cfg["width"]
    put("embed", cfg["vocab"], d, std=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        H, dim, vdim = mx["heads"], mx["dim"], mx["vdim"]
        put(p + "norm1", d, std=0.2)
        put(p + "norm1b", d, std=0.2)
        put(p + "mix.q", H * dim, d)
        put(p + "mix.o", d, H * vdim)
        if L["type"] == "gla":
            put(p + "mix.k", H * dim, d)
            put(p + "mix.v", H * vdim, d)
            put(p + "mix.g", H * vdim, d)
            put(p + "mix.norm", vdim, std=0.2, mean=1.0)
            put(p + "mix.a1", rank, d)
            put(p + "mix.a2", H * dim, rank)
            put(p + "mix.a2.b", H * dim, std=1.5)
        else:
            put(p + "mix.g", H, d)
            if mx.get("kv_from") is None:
                put(p + "mix.k", mx["kv_heads"] * dim, d)
                put(p + "mix.v", mx["kv_heads"] * vdim, d)
        if L.get("mlp") is not None:
            put(p + "norm2", d, std=0.2)
            put(p + "norm2b", d, std=0.2)
            put(p + "mlp.up", L["mlp"]["ff"], d)
            put(p + "mlp.down", d, L["mlp"]["ff"])
    put("final.norm", d, std=0.2)
    put("head", cfg["vocab"], d, std=4.0 * d ** -0.5)
    return W


def save_model(folder, cfg, W):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), W)
    return folder
