"""Plain, slow implementation of the Tekosun design, one function per mechanism, for comparison with the framework.

Written from the equations alone: torch tensors on the CPU, in the dtype the caller picks (float64 or float32), one sequence at
a time, token by token where a layer is recurrent, and nothing imported from the package.  ``W`` is a dict of tensors by their names in a checkpoint.
"""
import math

import torch

from folirax_ref import load, read_safetensors, save_model, write_safetensors  # noqa: F401  (the container, and nothing of a model)


# ---------------------------------------------------------------- norms and activations
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


def group_rms_norm(x, w, groups, eps):
    """Equal parts of a row, each over its own root mean square."""
    return unit_rms(x.view(*x.shape[:-1], groups, -1), eps).reshape(x.shape) * w


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


# ---------------------------------------------------------------- generalized delta rule
def delta_decay(h, w1, w2, w0):
    """Per head and key channel: exp(-e^(-1/2) sigmoid(low-rank projection + w0))."""
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(torch.tanh(h @ w1.T) @ w2.T + w0))


def unit_key(k):
    """k [..., dim] over its length."""
    return k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)


def delta_step(S, w, a, k, v):
    """S [H, dim, vdim]; w, a, k [H, dim]; v [H, vdim]."""
    u = unit_key(k)
    read = torch.einsum("hd,hdv->hv", u, S)
    return w[..., None] * S - (a * u)[..., None] * read[:, None, :] + k[..., None] * v[:, None, :]


def delta_rule(r, w, a, k, v, S):
    """All [T, H, dim]; returns (o [T, H, dim], the state behind the last token)."""
    out = []
    for t in range(r.shape[0]):
        S = delta_step(S, w[t], a[t], k[t], v[t])
        out.append(torch.einsum("hd,hdv->hv", r[t], S))
    return torch.stack(out), S


def delta_mixer(h, W, p, mx, eps, states, layer):
    T, H, D = h.shape[0], mx["heads"], mx["dim"]
    r, k, v = ((h @ W[p + n].T).view(T, H, D) for n in ("r", "k", "v"))
    w = delta_decay(h, W[p + "w1"], W[p + "w2"], W[p + "w0"]).view(T, H, D)
    a = torch.sigmoid(h @ W[p + "a"].T + W[p + "a.b"]).view(T, H, D)
    S = states.get(layer)
    o, states[layer] = delta_rule(r, w, a, k, v, torch.zeros(H, D, D, dtype=h.dtype) if S is None else S)
    o = unit_rms(o, eps).reshape(T, H * D) * W[p + "norm"]
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


# ---------------------------------------------------------------- Mamba-2
def causal_conv(x, before, w, b):
    """x [T, C] behind ``before`` [taps - 1, C]: every channel's own filter w [C, taps], the last tap on the current token.  Returns the result and the
    inputs the next call needs."""
    taps = w.shape[1]
    full = torch.cat([before, x])
    y = sum(full[i: i + x.shape[0]] * w[:, i] for i in range(taps)) + b
    return y, full[full.shape[0] - (taps - 1):]


def ssd(x, B, C, dt, A_log, D, S):
    """x [T, H, P], B and C [T, G, N], dt [T, H]; S [H, N, P].  Returns (y [T, H, P], state)."""
    T, H, _ = x.shape
    rep = H // B.shape[1]
    out = []
    for t in range(T):
        b, c = B[t].repeat_interleave(rep, 0), C[t].repeat_interleave(rep, 0)
        S = torch.exp(-torch.exp(A_log) * dt[t])[:, None, None] * S + dt[t][:, None, None] * b[..., None] * x[t][:, None, :]
        out.append(torch.einsum("hn,hnp->hp", c, S) + D[:, None] * x[t])
    return torch.stack(out), S


def mamba_mixer(h, W, p, mx, eps, states, layer):
    T, H, P, N, G = h.shape[0], mx["heads"], mx["vdim"], mx["state"], mx["groups"]
    inner = H * P
    z, xbc, dt = (h @ W[p + "in"].T).split([inner, inner + 2 * G * N, H], -1)
    before, S = states.get(layer) or (h.new_zeros(mx["conv"] - 1, inner + 2 * G * N), h.new_zeros(H, N, P))
    xbc, before = causal_conv(xbc, before, W[p + "conv"], W[p + "conv.b"])
    x, B, C = silu(xbc).split([inner, G * N, G * N], -1)
    y, S = ssd(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"], S)
    states[layer] = (before, S)
    return group_rms_norm(y.reshape(T, inner) * silu(z), W[p + "norm"], mx["norm_groups"], eps) @ W[p + "o"].T


# ---------------------------------------------------------------- attention
def frequencies(dims, base, scaling):
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f
    out = []
    for x in f:
        wave = 2 * math.pi / x
        if wave < scaling["original"] / scaling["high"]:
            out.append(x)
        elif wave > scaling["original"] / scaling["low"]:
            out.append(x / scaling["factor"])
        else:
            s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
            out.append((1 - s) * x / scaling["factor"] + s * x)
    return out


def rotate(x, pos, rot):
    """x [T, H, dim]: dimension i of the first ``dims`` turns with i + dims / 2."""
    n = rot["dims"] // 2
    a = torch.tensor(pos, dtype=torch.float64)[:, None] * torch.tensor(frequencies(rot["dims"], rot["base"], rot.get("scaling")), dtype=torch.float64)[None]
    c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
    u, v = x[..., :n], x[..., n: 2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def visible(first_pos, T, S, window):
    i, j = (first_pos + torch.arange(T))[:, None], torch.arange(S)[None, :]
    ok = j <= i
    return ok & (i - j < window) if window else ok


def attention(q, k, v, scale, window, first_pos):
    """q [T, H, dim] at first_pos.., k [S, G, dim], v [S, G, vdim]: [T, H, vdim]."""
    T, H = q.shape[:2]
    S, G = k.shape[:2]
    ok = visible(first_pos, T, S, window)
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~ok, -math.inf)
        out.append(torch.softmax(s, -1) @ v[:, g])
    return torch.stack(out, 1)


def mix_values(v, first, lam):
    return (1 - lam) * v + lam * first


def attention_mixer(h, W, p, mx, eps, pos0, cache, layer, shared):
    """``shared``: a dict that takes the first mixing layer's values of these tokens to the later ones."""
    T, H, G, D, V = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    pos = list(range(pos0, pos0 + T))
    q = rms_norm(h @ W[p + "q"].T, W[p + "q.norm"], eps).view(T, H, D)
    k = rms_norm(h @ W[p + "k"].T, W[p + "k.norm"], eps).view(T, G, D)
    v = unit_rms((h @ W[p + "v"].T).view(T, G, V), eps)
    q, k = rotate(q, pos, mx["rot"]), rotate(k, pos, mx["rot"])
    if mx.get("v_mix"):
        if "v" in shared:
            v = mix_values(v, shared["v"], W[p + "vmix"].reshape(()))
        else:
            shared["v"] = v
    if layer in cache:
        k, v = torch.cat([cache[layer][0], k]), torch.cat([cache[layer][1], v])
    cache[layer] = (k, v)
    window = mx["mask"]["size"] if mx.get("mask") else 0
    return attention(q, k, v, mx["scale"], window, pos0).reshape(T, H * V) @ W[p + "o"].T


# ---------------------------------------------------------------- mixture of experts
def relu2_ff(h, W, p):
    return torch.relu(h @ W[p + "up"].T) ** 2 @ W[p + "down"].T


def route(h, router, top, scale):
    """Chosen experts and their weights, [T, top] each."""
    s = torch.softmax(h @ router.T, -1)
    w, e = s.topk(top, -1)
    return e, w / (w.sum(-1, keepdim=True) + 1e-20) * scale


def expert_ff(h, W, p, mlp):
    e, w = route(h, W[p + "router"], mlp["router"]["top"], mlp["router"]["scale"])
    out = relu2_ff(h, W, p + "shared.") if mlp.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for n in range(e.shape[1]):
            out[t] += w[t, n] * relu2_ff(h[t][None], W, f"{p}e{int(e[t, n])}.")[0]
    return out


# ---------------------------------------------------------------- the model
class Sequence:
    """What one sequence has left behind, per layer."""

    def __init__(self):
        self.cache, self.states, self.length = {}, {}, 0


def forward(cfg, W, tokens, seq, layers_out=None):
    """Append ``tokens``; logits [T, vocab] of every one.  ``layers_out``: a list that takes the residual behind every layer."""
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    shared = {}
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        if L["type"] == "general_delta":
            y = delta_mixer(x, W, p + "mix.", mx, eps, seq.states, i)
        elif L["type"] == "mamba2":
            y = mamba_mixer(x, W, p + "mix.", mx, eps, seq.states, i)
        else:
            y = attention_mixer(x, W, p + "mix.", mx, eps, seq.length, seq.cache, i, shared)
        x = x + rms_norm(y, W[p + "norm1"], eps)
        if L.get("mlp") is not None:
            x = x + rms_norm(expert_ff(x, W, p + "mlp.", L["mlp"]), W[p + "norm2"], eps)
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
def moe(ff, experts, top, scale=1.0, shared=24):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}, "shared": {"ff": shared} if shared else None}


def layer_delta(dim, heads, mlp=None):
    return {"type": "general_delta", "mixer": {"dim": dim, "heads": heads}, "mlp": mlp}


def layer_mamba(heads, vdim, state, groups=1, norm_groups=1, conv=4, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}, "mlp": mlp}


def layer_attention(dim, vdim, heads, kv_heads, rot_dims, window=0, base=10000.0, scaling=None, scale=None, v_mix=True, mlp=None):
    """``scaling``: (factor, low, high, original)."""
    rot = {"base": base, "dims": rot_dims}
    if scaling is not None:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return {"type": "attention", "mlp": mlp, "mixer": {"dim": dim, "vdim": vdim, "heads": heads, "kv_heads": kv_heads, "rot": rot, "v_mix": v_mix,
                                                       "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": window} if window else None}}


def config(layers, width, vocab, eps=1e-5, scale=1.0):
    return {"architecture": "Tekosun", "layers": layers, "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": scale}}


def random_weights(cfg, seed=0, rank=8):
    """Seeded weights, rounded to bf16 (what a checkpoint holds), returned in float64."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def put(name, *shape, std=None, mean=0.0):
        s = shape[-1] ** -0.5 if std is None else std
        W[name] = (torch.randn(shape, generator=g, dtype=torch.float64) * s + mean).to(torch.bfloat16).double()
    d = cfg["width"]
    put("embed", cfg["vocab"], d, std=1.0 / cfg["embedding"]["scale"])
    for i, L in enumerate(cfg["layers"]):
        p, mx, mlp = f"l{i}.", L["mixer"], L.get("mlp")
        put(p + "norm1", d, std=0.2, mean=0.8)
        if L["type"] == "general_delta":
            hd = mx["heads"] * mx["dim"]
            for n in ("r", "k", "v", "g", "a"):
                put(f"{p}mix.{n}", hd, d)
            put(p + "mix.a.b", hd, std=1.0, mean=0.5)
            put(p + "mix.w1", rank, d)
            put(p + "mix.w2", hd, rank, std=1.5 * rank ** -0.5)
            put(p + "mix.w0", hd, std=2.0, mean=-3.0)
            put(p + "mix.norm", hd, std=0.2, mean=1.0)
            put(p + "mix.o", d, hd)
        elif L["type"] == "mamba2":
            H, inner = mx["heads"], mx["heads"] * mx["vdim"]
            channels = inner + 2 * mx["groups"] * mx["state"]
            put(p + "mix.in", inner + channels + H, d, std=1.3 * d ** -0.5)
            put(p + "mix.conv", channels, mx["conv"], std=0.7)
            put(p + "mix.conv.b", channels, std=0.3)
            put(p + "mix.dt_bias", H, std=1.0, mean=-2.0)
            put(p + "mix.A_log", H, std=1.0)
            put(p + "mix.D", H, std=0.5, mean=0.5)
            put(p + "mix.norm", inner, std=0.2, mean=1.0)
            put(p + "mix.o", d, inner)
        else:
            H, G = mx["heads"], mx["kv_heads"]
            for n, rows in (("q", H * mx["dim"]), ("k", G * mx["dim"]), ("v", G * mx["vdim"])):
                put(f"{p}mix.{n}", rows, d)
            put(p + "mix.q.norm", H * mx["dim"], std=0.5, mean=1.5)
            put(p + "mix.k.norm", G * mx["dim"], std=0.5, mean=1.5)
            if mx["v_mix"]:
                W[p + "mix.vmix"] = torch.tensor(0.15 + 0.4 * torch.rand(1, generator=g).item(), dtype=torch.float64).to(torch.bfloat16).double()
            put(p + "mix.o", d, H * mx["vdim"])
        if mlp is not None:
            put(p + "norm2", d, std=0.2, mean=0.8)
            for e, ff in [(f"e{e}", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])] + ([("shared", mlp["shared"]["ff"])] if mlp["shared"] else []):
                put(f"{p}mlp.{e}.up", ff, d)
                put(f"{p}mlp.{e}.down", d, ff)
            put(p + "mlp.router", mlp["router"]["experts"], d, std=2.0 * d ** -0.5)
    put("final.norm", d, std=0.3, mean=1.0)
    put("head", cfg["vocab"], d, std=4.0 * d ** -0.5)
    return W
