"""Plain, slow implementation of the Kazolorn design, one function per mechanism, for comparison with the framework.

Written from the equations alone: torch tensors on the CPU, in the dtype the caller picks (float64 or float32), one sequence at
a time, and nothing imported from the package.  ``W`` is a dict of tensors by their names in a checkpoint.
"""
import math

import torch

from folirax_ref import load, read_safetensors, save_model, write_safetensors  # noqa: F401  (the container, and nothing of a model)


# ---------------------------------------------------------------- mechanisms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def slopes(H, dtype=torch.float64):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / H) for h in range(H)], dtype=dtype)


def raw_scores(q, k, scale):
    """q [T, H, dim], k [S, G, dim] -> [H, T, S]; query head h reads key head h // (H / G)."""
    T, H = q.shape[:2]
    rep = H // k.shape[1]
    return torch.stack([q[:, h] @ k[:, h // rep].T * scale for h in range(H)])


def distance_bias(s, first_pos):
    """Takes slope_h * (i - j) off; the queries stand at first_pos.., the keys at 0.."""
    H, T, S = s.shape
    i, j = (first_pos + torch.arange(T))[:, None], torch.arange(S)[None, :]
    return s - slopes(H, s.dtype)[:, None, None] * (i - j).to(s.dtype)


def talk(s, mix):
    """Every head's scores become a mixture of all heads': mix [H, H], row = the head that results."""
    return torch.einsum("hg,gts->hts", mix, s)


def visible(first_pos, T, S, window):
    i, j = (first_pos + torch.arange(T))[:, None], torch.arange(S)[None, :]
    return (j <= i) & (i - j < window)


def weights_with_silent_sink(s, ok):
    """exp(s) over one plus the sum of exp(s) over the visible keys."""
    s = s.masked_fill(~ok[None], -math.inf)
    m = s.amax(-1, keepdim=True).clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attention(q, k, mix, scale, window, first_pos):
    """q [T, H, dim] at first_pos.., k [S, G, dim]: [T, H, dim]; the keys are the values too."""
    T, H = q.shape[:2]
    S, G = k.shape[:2]
    s = talk(distance_bias(raw_scores(q, k, scale), first_pos), mix)
    p = weights_with_silent_sink(s, visible(first_pos, T, S, window))
    return torch.stack([p[h] @ k[:, h // (H // G)] for h in range(H)], 1)


def attention_mixer(h, W, p, mx, pos0, cache, layer):
    T, H, G, dim = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, dim)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, dim)
    cache[layer] = torch.cat([cache[layer], k]) if layer in cache else k
    o = attention(q, cache[layer], W[p + "talk"], mx["scale"], mx["mask"]["size"], pos0)
    return o.reshape(T, H * dim) @ W[p + "o"].T + W[p + "o.b"]


def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * unit_rms(z, eps) + b * unit_rms(z ** 2, eps) + c * unit_rms(z ** 3, eps) + e


def dense_ff(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def route(h, router, top):
    """Chosen experts and their weights, [T, top] each: the largest sigmoid scores, as they are."""
    s = torch.sigmoid(h @ router.T)
    w, e = s.topk(top, -1)
    return e, w


def expert(h, W, p):
    g = h @ W[p + "gate"].T
    return (g * torch.sigmoid(g) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def expert_ff(h, W, p, top):
    """The weight scales what goes into an expert."""
    e, w = route(h, W[p + "router"], top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for n in range(top):
            out[t] += expert((w[t, n] * h[t])[None], W, f"{p}e{int(e[t, n])}.")[0]
    return out


def depth_average(xs, weights):
    return sum(w * x for w, x in zip(weights, xs))


class Sequence:
    """What one sequence has left behind, per layer."""

    def __init__(self):
        self.cache, self.length = {}, 0


def forward(cfg, W, tokens, seq, layers_out=None):
    """Append ``tokens``; logits [T, vocab] of every one.  ``layers_out``: a list that takes the residual behind every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    xs = [x]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = x + W[p + "ls1"] * attention_mixer(rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", L["mixer"], seq.length, seq.cache, i)
        if L.get("mlp") is not None:
            h = rms_norm(x, W[p + "norm2"], eps)
            ff = dense_ff(h, W, p + "mlp.", eps) if L["mlp"]["kind"] == "dense" else expert_ff(h, W, p + "mlp.", L["mlp"]["router"]["top"])
            y = y + W[p + "ls2"] * ff
        xs.append(y)
        x = depth_average(xs, W[p + "dwa"])
        if layers_out is not None:
            layers_out.append(x.clone())
    seq.length += len(tokens)
    return rms_norm(x, W["final.norm"], eps) @ W["head"].T


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
def layer(dim, heads, kv_heads, window, ff=None, experts=None, top=1, scale=None):
    """``experts``: a mixture of that many feed-forwards of width ``ff`` instead of one."""
    mlp = None
    if experts is not None:
        mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    elif ff is not None:
        mlp = {"kind": "dense", "ff": ff}
    mx = {"dim": dim, "vdim": dim, "heads": heads, "kv_heads": kv_heads, "mask": {"size": window}, "scale": dim ** -0.5 if scale is None else scale}
    return {"type": "attention", "mixer": mx, "mlp": mlp}


def config(layers, width, vocab, eps=1e-5):
    return {"architecture": "Kazolorn", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}}


def random_weights(cfg, seed=0):
    """Seeded weights, rounded to bf16 (what a checkpoint holds), returned in float64."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def put(name, *shape, std=None, mean=0.0):
        s = shape[-1] ** -0.5 if std is None else std
        W[name] = (torch.randn(shape, generator=g, dtype=torch.float64) * s + mean).to(torch.bfloat16).double()
    d = cfg["width"]
    put("embed", cfg["vocab"], d, std=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        H, G, dim = mx["heads"], mx["kv_heads"], mx["dim"]
        put(p + "norm1", d, std=0.3, mean=1.0)
        for n, rows in (("q", H * dim), ("k", G * dim)):
            put(p + "mix." + n, rows, d, std=1.2 * d ** -0.5)
            put(p + "mix." + n + ".b", rows, std=0.4)
        put(p + "mix.talk", H, H, std=0.6 * H ** -0.5)
        W[p + "mix.talk"] = (W[p + "mix.talk"] + torch.eye(H, dtype=torch.float64)).to(torch.bfloat16).double()
        put(p + "mix.o", d, H * dim)
        put(p + "mix.o.b", d, std=0.2)
        put(p + "ls1", d, std=0.2, mean=0.7)
        if mlp is not None:
            put(p + "norm2", d, std=0.3, mean=1.0)
            put(p + "ls2", d, std=0.2, mean=0.8)
            if mlp["kind"] == "dense":
                put(p + "mlp.up", mlp["ff"], d, std=1.5 * d ** -0.5)
                put(p + "mlp.down", d, mlp["ff"])
                put(p + "mlp.act", 4, std=0.3, mean=0.5)
            else:
                for e in range(mlp["router"]["experts"]):
                    put(f"{p}mlp.e{e}.gate", mlp["expert"]["ff"], d, std=2.0 * d ** -0.5)
                    put(f"{p}mlp.e{e}.up", mlp["expert"]["ff"], d, std=2.0 * d ** -0.5)
                    put(f"{p}mlp.e{e}.down", d, mlp["expert"]["ff"])
                put(p + "mlp.router", mlp["router"]["experts"], d, std=2.0 * d ** -0.5)
        put(p + "dwa", i + 2, std=0.3, mean=0.1)
        W[p + "dwa"][-1] += 0.8
        W[p + "dwa"] = W[p + "dwa"].to(torch.bfloat16).double()
    put("final.norm", d, std=0.3, mean=1.0)
    put("head", cfg["vocab"], d, std=4.0 * d ** -0.5)
    return W
