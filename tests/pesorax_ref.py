"""Plain, slow implementation of the Pesorax design, one function per mechanism, for comparison with the framework.

Written from the equations alone: torch tensors on the CPU, in the dtype the caller picks (float64 or float32), one sequence at
a time, and nothing imported from the package.  ``W`` is a dict of tensors by their names in a checkpoint.
"""
import math

import torch

from folirax_ref import load, read_safetensors, save_model, write_safetensors  # noqa: F401  (the container, and nothing of a model)


# ---------------------------------------------------------------- mechanisms
def dyt(x, W, name):
    """Dynamic Tanh: a squashed scale and shift per channel, no statistics of the row."""
    return torch.tanh(W[name + ".alpha"] * x) * W[name] + W[name + ".b"]


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rotate_half(x, pos, dims, base):
    """x [T, heads, dim]: dimension i turns with i + dims/2 by the angle pos * base^(-2i/dims); the rest stays."""
    out = x.clone()
    n = dims // 2
    for i in range(n):
        a = (pos.to(torch.float64) * float(base) ** (-2.0 * i / dims)).to(x.dtype)[:, None]
        c, s = torch.cos(a), torch.sin(a)
        u, v = x[..., i], x[..., i + n]
        out[..., i] = u * c - v * s
        out[..., i + n] = v * c + u * s
    return out


def visible(first_pos, T, S, chunk=0):
    """[T, S]: which keys (positions 0..S-1) the queries at first_pos.. see; ``chunk``: only those of their own chunk."""
    i, j = (first_pos + torch.arange(T))[:, None], torch.arange(S)[None, :]
    ok = j <= i
    if chunk:
        ok = ok & (i // chunk == j // chunk)
    return ok


def weights_over_keys(s, ok, sink=None):
    """Softmax over the visible keys of s [H, T, S]; ``sink`` [H]: one more term of the denominator per head."""
    s = s.masked_fill(~ok[None], -math.inf)
    m = s.amax(-1, keepdim=True)
    if sink is not None:
        m = torch.maximum(m, sink[:, None, None])
    e = torch.exp(s - m)
    z = e.sum(-1, keepdim=True)
    if sink is not None:
        z = z + torch.exp(sink[:, None, None] - m)
    return e / z


def lambda_of(W, p, diff):
    """The weight of the second map: one number for the layer."""
    return torch.exp((W[p + "lq1"] * W[p + "lk1"]).sum()) - torch.exp((W[p + "lq2"] * W[p + "lk2"]).sum()) + diff


def differential_attention(q, k, v, scale, chunk, first_pos):
    """q [T, H, 2, dim], k [S, G, 2, dim], v [S, G, vdim]: the outputs of both maps, [2][T, H, vdim]."""
    T, H = q.shape[:2]
    S, G = k.shape[:2]
    ok = visible(first_pos, T, S, chunk)
    outs = []
    for m in range(2):
        o = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
        for h in range(H):
            g = h // (H // G)
            s = (q[:, h, m] @ k[:, g, m].T * scale)[None]
            o[:, h] = weights_over_keys(s, ok)[0] @ v[:, g]
        outs.append(o)
    return outs


def differential_mixer(h, W, p, mx, eps, pos0, cache, run):
    T = h.shape[0]
    H, G, dim, vdim = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, 2, dim)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, 2, dim)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(T, G, vdim)
    old = cache.get(run)
    cache[run] = (k, v) if old is None else (torch.cat([old[0], k]), torch.cat([old[1], v]))
    a1, a2 = differential_attention(q, *cache[run], mx["scale"], mx["mask"]["size"], pos0)
    o = unit_rms(a1 - lambda_of(W, p, mx["diff"]) * a2, eps) * (1 - mx["diff"])
    return o.reshape(T, H * vdim) @ W[p + "o"].T


def latent_mixer(h, W, p, mx, eps, pos0, cache, run):
    """Keys and values come out of a shared latent; what is kept per token is that latent and one rotated key part."""
    T = h.shape[0]
    H, dim, rd, vdim, rank = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = torch.arange(pos0, pos0 + T)
    rot = lambda x: rotate_half(x, pos, mx["rot"]["dims"], mx["rot"]["base"])       # noqa: E731
    cq = unit_rms(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    q = (cq @ W[p + "uq"].T).view(T, H, dim + rd)
    qn, qr = q[..., :dim], rot(q[..., dim:])
    kv = h @ W[p + "dkv"].T
    c = unit_rms(kv[:, :rank], eps) * W[p + "dkv.norm"]
    kr = rot(kv[:, None, rank:])[:, 0]
    old = cache.get(run)
    cache[run] = (c, kr) if old is None else (torch.cat([old[0], c]), torch.cat([old[1], kr]))
    c, kr = cache[run]
    S = c.shape[0]
    kn = (c @ W[p + "uk"].T).view(S, H, dim)
    v = (c @ W[p + "uv"].T).view(S, H, vdim)
    s = (torch.einsum("thd,shd->hts", qn, kn) + torch.einsum("thr,sr->hts", qr, kr)) * mx["scale"]
    w = weights_over_keys(s, visible(pos0, T, S), W[p + "sink"])
    o = torch.einsum("hts,shv->thv", w, v).reshape(T, H * vdim)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def gelu_ff(h, W, p):
    z = h @ W[p + "up"].T
    return (0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))) @ W[p + "down"].T


def order(cfg):
    """Layer runs in order: (layer, whether the embedding output joins ahead of it)."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


class Sequence:
    """What one sequence has left behind, per layer run."""

    def __init__(self):
        self.cache, self.length = {}, 0


def forward(cfg, W, tokens, seq, layers_out=None):
    """Append ``tokens``; logits [T, vocab] of every one.  ``layers_out``: a list that takes the residual after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    emb = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    x = emb
    for run, (i, joins) in enumerate(order(cfg)):
        p, L = f"l{i}.", cfg["layers"][i]
        if joins:
            x = x + emb
        mixer = {"attention": differential_mixer, "latent_attention": latent_mixer}[L["type"]]
        x = x + m * mixer(dyt(x, W, p + "norm1"), W, p + "mix.", L["mixer"], eps, seq.length, seq.cache, run)
        if L.get("mlp") is not None:
            x = x + m * gelu_ff(dyt(x, W, p + "norm2"), W, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    seq.length += len(tokens)
    return dyt(x, W, "final.norm") @ W["head"].T


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
def layer_attention(dim, vdim, heads, kv_heads, chunk, diff=0.4, scale=None, ff=None):
    mx = {"dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": chunk}, "diff": diff,
          "scale": dim ** -0.5 if scale is None else scale}
    return {"type": "attention", "mixer": mx, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def layer_latent(dim, rot_dim, vdim, heads, kv_rank, q_rank, base=10000.0, scale=None, ff=None):
    mx = {"dim": dim, "rot_dim": rot_dim, "vdim": vdim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank,
          "rot": {"base": base, "dims": rot_dim}, "scale": (dim + rot_dim) ** -0.5 if scale is None else scale}
    return {"type": "latent_attention", "mixer": mx, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, loop=None, eps=1e-5, residual_mult=0.6):
    c = {"architecture": "Pesorax", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": residual_mult}
    if loop is not None:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def random_weights(cfg, seed=0):
    """Seeded weights, rounded to bf16 (what a checkpoint holds), returned in float64."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def put(name, *shape, std=None, mean=0.0):
        s = shape[-1] ** -0.5 if std is None else std
        W[name] = (torch.randn(shape, generator=g, dtype=torch.float64) * s + mean).to(torch.bfloat16).double()

    def norm(name):
        put(name, d, std=0.3, mean=1.0)
        put(name + ".b", d, std=0.2)
        put(name + ".alpha", std=0.1, mean=0.8)
    d = cfg["width"]
    put("embed", cfg["vocab"], d, std=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        H, dim, vdim = mx["heads"], mx["dim"], mx["vdim"]
        norm(p + "norm1")
        if L["type"] == "attention":
            G = mx["kv_heads"]
            for n, rows in (("q", 2 * H * dim), ("k", 2 * G * dim), ("v", G * vdim)):
                put(p + "mix." + n, rows, d, std=1.5 * d ** -0.5)
                put(p + "mix." + n + ".b", rows, std=0.5)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                put(p + "mix." + n, dim, std=0.6 * dim ** -0.25)
        else:
            put(p + "mix.dq", mx["q_rank"], d)
            put(p + "mix.dq.norm", mx["q_rank"], std=0.2, mean=1.0)
            put(p + "mix.uq", H * (dim + mx["rot_dim"]), mx["q_rank"], std=2.0 * mx["q_rank"] ** -0.5)
            put(p + "mix.dkv", mx["kv_rank"] + mx["rot_dim"], d)
            put(p + "mix.dkv.norm", mx["kv_rank"], std=0.2, mean=1.0)
            put(p + "mix.uk", H * dim, mx["kv_rank"], std=1.5 * mx["kv_rank"] ** -0.5)
            put(p + "mix.uv", H * vdim, mx["kv_rank"])
            put(p + "mix.sink", H, std=1.0, mean=1.0)
            put(p + "mix.g", H * vdim, d, std=2.0 * d ** -0.5)
        put(p + "mix.o", d, H * vdim)
        if L.get("mlp") is not None:
            norm(p + "norm2")
            put(p + "mlp.up", L["mlp"]["ff"], d, std=1.5 * d ** -0.5)
            put(p + "mlp.down", d, L["mlp"]["ff"])
    norm("final.norm")
    put("head", cfg["vocab"], d, std=4.0 * d ** -0.5)
    return W
