"""Plain statements of the Bugipel design's mechanisms (PyTorch, any dtype; the tests use float64), one function each, and a
whole-model forward that recomputes every position from the full token list.  Nothing here is shared with the package:
weights come in as a dict of tensors under the checkpoint's names, the configuration as the parsed config.json.

The design: pre-norm layers (RMS norms with a weight vector), some of which run several times in a row with the same weights; in
front of every pass the stream is projected back from [stream ; embedding output] and a vector of the pass's own is added.  Mixers:
lightning attention (a linear recurrence with one constant decay per head, silu on q, k and v, a norm over all heads together
under a sigmoid gate), and "parallel": softmax attention whose values are its un-normalised, un-rotated keys, with unit-RMS
queries and keys behind the rotation, a one in the softmax's denominator and a gate per channel -- beside a delta rule whose state
decays per key channel; the two are added with a scale each.  Feed-forward: down(gelu(up h)).  The head is the embedding table.
"""
import math

import torch


# ------------------------------------------------------------------ small pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def softplus(z):
    return torch.where(z > 30, z, torch.log1p(torch.exp(torch.clamp(z, max=30))))


def causal_taps(h, w):
    """h [T, C], w [C, taps] (last column multiplies the current token), zeros before the first token"""
    T, C = h.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=h.dtype), h], dim=0)
    out = torch.zeros_like(h)
    for j in range(taps):
        out = out + padded[j:j + T] * w[:, j]
    return out


def rotate_half(x, positions, dims, base):
    """x [T, heads, D]: channel i < dims / 2 of every head is rotated with channel i + dims / 2 by position * base^(-2i / dims)"""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    ang = positions.to(x.dtype)[:, None] * f[None, :]
    cos, sin = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    a, b = x[..., :half], x[..., half:dims]
    return torch.cat([a * cos - b * sin, b * cos + a * sin, x[..., dims:]], dim=-1)


# ------------------------------------------------------------------ attention
def softmax_with_one(s):
    """exp(s) / (1 + sum exp(s)) over the last axis"""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def visible_attention(q, k, v, scale, held=0, first=0, sink=True):
    """q [S, H, D]: new tokens that sit at indices held .. held + S - 1 of k [L, G, D] / v [L, G, Dv]; indices below ``first`` do not
    exist (padding).  Returns [S, H, Dv] (zeros where no query exists)."""
    S, H, D = q.shape
    per = H // k.shape[1]
    out = torch.zeros(S, H, v.shape[2], dtype=q.dtype)
    for t in range(S):
        c = held + t
        if c < first:
            continue
        for hd in range(H):
            s = (k[first:c + 1, hd // per] @ q[t, hd]) * scale
            out[t, hd] = (softmax_with_one(s) if sink else torch.softmax(s, dim=0)) @ v[first:c + 1, hd // per]
    return out


def prepare_qk(q, k, positions, rot, eps):
    """queries and keys [T, heads, D]: rotated, then divided by their root mean square per head (no weight)"""
    dims, base = int(rot["dims"]), float(rot["base"])
    return unit_rms(rotate_half(q, positions, dims, base), eps), unit_rms(rotate_half(k, positions, dims, base), eps)


def key_value_attention(h, W, m, eps):
    """the attention branch: keys are the values"""
    T = h.shape[0]
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    v = (h @ W["k"].T).view(T, G, D)
    q, k = prepare_qk((h @ W["q"].T).view(T, H, D), v, torch.arange(T), m["rot"], eps)
    k, v = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q, k) * float(m["scale"])
    s = s.masked_fill(~torch.tril(torch.ones(T, T, dtype=torch.bool))[None], float("-inf"))
    o = torch.einsum("hij,jhd->ihd", softmax_with_one(s), v).reshape(T, H * D)
    return (o * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


# ------------------------------------------------------------------ recurrences
def channel_decay(h, W, H, D):
    """per head and key channel, in (0, 1)"""
    dt = softplus((h @ W["a1"].T) @ W["a2"].T + W["dt_bias"]).view(h.shape[0], H, D)
    return torch.exp(-torch.exp(W["A_log"]).view(1, H, 1) * dt)


def channel_delta_scan(q, k, v, g, beta):
    """q, k, g [T, H, D]; v [T, H, Dv]; beta [T, H].  State S [H, D, Dv] from zero:
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q"""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t].unsqueeze(-1) * S
        u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(-2)
        out.append(torch.einsum("hij,hi->hj", S, q[t]))
    return torch.stack(out)


def channel_delta_branch(h, W, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    assert W["q.conv"].shape[1] == int(m["conv"])
    q = silu(causal_taps(h @ W["q"].T, W["q.conv"])).view(T, G, D)
    k = silu(causal_taps(h @ W["k"].T, W["k.conv"])).view(T, G, D)
    v = silu(causal_taps(h @ W["v"].T, W["v.conv"])).view(T, H, Dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * D ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    o = channel_delta_scan(q, k, v, channel_decay(h, W, H, D), torch.sigmoid(h @ W["b"].T))
    o = unit_rms(o, eps) * W["norm"] * torch.sigmoid((h @ W["g1"].T) @ W["g2"].T).view(T, H, Dv)
    return o.reshape(T, H * Dv) @ W["o"].T


def constant_decay_scan(q, k, v, decay):
    """q, k [T, H, D]; v [T, H, Dv]; decay [H].  S <- decay S + k v^T;  o = S^T q"""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = decay.view(H, 1, 1) * S + k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        out.append(torch.einsum("hij,hi->hj", S, q[t]))
    return torch.stack(out)


# ------------------------------------------------------------------ mixers
def lightning_mixer(h, W, m, eps):
    T = h.shape[0]
    H, D, Dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = silu(h @ W["q"].T).view(T, H, D), silu(h @ W["k"].T).view(T, H, D), silu(h @ W["v"].T).view(T, H, Dv)
    o = constant_decay_scan(q, k, v, torch.tensor(m["decay"], dtype=h.dtype)).reshape(T, H * Dv)
    return (unit_rms(o, eps) * W["norm"] * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


def parallel_mixer(h, W, m, eps):
    left = key_value_attention(h, sub(W, "left."), m["left"], eps)
    right = channel_delta_branch(h, sub(W, "right."), m["right"], eps)
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


MIXERS = {"lightning": lightning_mixer, "parallel": parallel_mixer}


# ------------------------------------------------------------------ the model
def sub(weights, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in weights.items() if k.startswith(prefix)}


def layer_runs(cfg):
    """(layer, number of the pass whose first layer this is or None) in the order in which layers run"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t if i == a else None) for i in range(a, b)]
    return runs + [(i, None) for i in range(b, n)]


def enter_pass(x, x0, weights, t):
    return torch.cat([x, x0], dim=-1) @ weights["loop.in"].T + weights["loop.step"][t]


def forward(cfg, weights, tokens, collect=None):
    """logits [T, vocab] of one sequence; ``collect``: a list that receives the stream after every layer run"""
    eps = float(cfg["norm"]["eps"])
    x0 = x = weights["embed"][torch.as_tensor(tokens)]
    for i, t in layer_runs(cfg):
        if t is not None:
            x = enter_pass(x, x0, weights, t)
        lc, W = cfg["layers"][i], sub(weights, f"l{i}.")
        x = x + MIXERS[lc["type"]](unit_rms(x, eps) * W["norm1"], sub(W, "mix."), lc["mixer"], eps)
        if lc.get("mlp") is not None:
            h = unit_rms(x, eps) * W["norm2"]
            x = x + gelu_erf(h @ W["mlp.up"].T) @ W["mlp.down"].T
        if collect is not None:
            collect.append(x.clone())
    return (unit_rms(x, eps) * weights["final.norm"]) @ weights["embed"].T


def greedy(cfg, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens


# ------------------------------------------------------------------ random models
LIGHT = dict(heads=3, dim=10, vdim=14, decay=None)
LEFT = dict(heads=6, kv_heads=2, dim=12, rot_dims=8, base=50.0, scale=0.4)
RIGHT = dict(heads=4, kv_heads=2, dim=6, vdim=10, conv=3)


def random_config(width=40, vocab=61, order=("parallel", "lightning", "parallel", "lightning"), ffs=(24, 56, None, 33), light=None, left=None,
                  right=None, loop=(1, 3, 3), scales=(0.7, 1.3), eps=1e-5):
    """``order``: the layers' mixers; ``ffs``: per layer the feed-forward's width or None; the dicts override the sizes above;
    ``loop``: (start, stop, times) or None"""
    li, le, ri = (dict(base, **(over or {})) for base, over in ((LIGHT, light), (LEFT, left), (RIGHT, right)))
    decay = li["decay"] or [1.0 - 0.5 / (1 + 2 * h) ** 2 for h in range(li["heads"])]
    layers = []
    for kind, ff in zip(order, ffs):
        if kind == "lightning":
            mixer = {"heads": li["heads"], "dim": li["dim"], "vdim": li["vdim"], "decay": decay}
        else:
            mixer = {"left": {"heads": le["heads"], "kv_heads": le["kv_heads"], "dim": le["dim"], "vdim": le["dim"], "scale": le["scale"],
                              "rot": {"base": le["base"], "dims": le["rot_dims"]}}, "left_scale": scales[0],
                     "right": {k: ri[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv")}, "right_scale": scales[1]}
        layers.append({"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}})
    cfg = {"architecture": "Bugipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed, ranks=(5, 3), dtype=torch.bfloat16):
    """weights under the checkpoint's names; ``ranks``: the inner sizes of the delta rule's decay and gate projections"""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def vec(n, mean=1.0, s=0.2):
        return mean + torch.randn(n, generator=g) * s

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g), "final.norm": vec(W)}
    if cfg.get("loop"):
        w["loop.in"], w["loop.step"] = mat(W, 2 * W, 1.3), torch.randn(cfg["loop"]["times"], W, generator=g) * 0.4
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        w[p + "norm1"] = vec(W)
        x = p + "mix."
        if lc["type"] == "lightning":
            H, D, Dv = m["heads"], m["dim"], m["vdim"]
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                w[x + n] = mat(rows, W, 1.5)
            w[x + "norm"], w[x + "o"] = vec(H * Dv), mat(W, H * Dv)
        else:
            l, r = m["left"], m["right"]
            H, G, D = l["heads"], l["kv_heads"], l["dim"]
            w[x + "left.q"], w[x + "left.k"], w[x + "left.g"] = mat(H * D, W, 2.0), mat(G * D, W, 1.5), mat(H * D, W)
            w[x + "left.o"] = mat(W, H * D)
            H, G, D, Dv, T = r["heads"], r["kv_heads"], r["dim"], r["vdim"], r["conv"]
            x += "right."
            for n, rows in (("q", G * D), ("k", G * D), ("v", H * Dv)):
                w[x + n], w[x + n + ".conv"] = mat(rows, W, 2.0), torch.randn(rows, T, generator=g) * 0.6
            w[x + "b"] = mat(H, W, 2.0)
            w[x + "a1"], w[x + "a2"] = mat(ranks[0], W), mat(H * D, ranks[0], 2.0)
            w[x + "g1"], w[x + "g2"] = mat(ranks[1], W), mat(H * Dv, ranks[1], 2.0)
            w[x + "A_log"], w[x + "dt_bias"] = torch.randn(H, generator=g) * 0.7 - 0.5, torch.randn(H * D, generator=g) - 1.0
            w[x + "norm"], w[x + "o"] = vec(Dv), mat(W, H * Dv)
        if lc.get("mlp") is not None:
            F = lc["mlp"]["ff"]
            w[p + "norm2"], w[p + "mlp.up"], w[p + "mlp.down"] = vec(W), mat(F, W, 2.0), mat(W, F)
    return {k: v.to(dtype) for k, v in w.items()}
