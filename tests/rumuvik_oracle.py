"""Plain statements of the Rumuvik design's mechanisms (PyTorch, any dtype; the tests use float64), one function each, and a
whole-model forward that recomputes every position from the full token list.  Nothing here is shared with the package:
weights come in as a dict of tensors under the checkpoint's names, the configuration as the parsed config.json.

The design: layers whose mixer and feed-forward read two RMS norms (weights stored around zero) of the same stream and are added to
it together; a stretch of the layers runs several times with the same weights, the embedding output being added in front of every
pass but the first.  Mixers: grouped attention whose VALUES are rotated by their own position and whose output is turned back by the
query's, with capped scores and a one in the softmax's denominator; latent attention with a query latent and one rotated key part
that all heads share; the matrix memory of an mLSTM (exponential input gate, running maximum, normaliser).  Feed-forward:
down(gelu_tanh(gate h) * up h).
"""
import math

import torch


# ------------------------------------------------------------------ small pieces
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, w, eps):
    return unit_rms(x, eps) * (1.0 + w)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def cap_scores(s, cap):
    return cap * torch.tanh(s / cap)


def softmax_with_one(s):
    """exp(s) / (1 + sum exp(s)) over the last axis"""
    top = torch.clamp(s.max(-1, keepdim=True).values, min=0.0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def sub(weights, prefix):
    n = len(prefix)
    return {k[n:]: v for k, v in weights.items() if k.startswith(prefix)}


# ------------------------------------------------------------------ positions
def plain_frequencies(dims, base, dtype=torch.float64):
    return torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=dtype)


def rot_frequencies(rot, dtype=torch.float64):
    """(frequencies, amplitude) of a ``rot`` block; with ``scaling`` slow pairs turn ``factor`` times slower, fast ones as before"""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = plain_frequencies(dims, base, dtype)
    sc = rot.get("scaling")
    if sc is None:
        return f, 1.0

    def where(turns):
        return dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))

    lo, hi = max(math.floor(where(sc["fast"])), 0), min(math.ceil(where(sc["slow"])), dims - 1)
    i = torch.arange(dims // 2, dtype=dtype)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / sc["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def turn(x, positions, freq, amp=1.0, interleaved=False, back=False):
    """x [T, heads, D]: pair i of the first 2 * len(freq) channels is turned by position * freq[i] (by minus that with ``back``); pairs
    are (i, i + n), or (2i, 2i + 1) when ``interleaved``; the other channels pass"""
    n = len(freq)
    a = positions.to(x.dtype)[:, None] * freq.to(x.dtype)[None, :] * (-1.0 if back else 1.0)
    c, s = (torch.cos(a) * amp)[:, None, :], (torch.sin(a) * amp)[:, None, :]
    y = x.clone()
    first, second = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if interleaved else (slice(0, n), slice(n, 2 * n))
    u, v = x[..., first], x[..., second]
    y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y


# ------------------------------------------------------------------ mixers
def causal(T):
    return torch.tril(torch.ones(T, T, dtype=torch.bool))


def turned_value_attention(q, k, v, positions, rot, scale, cap):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] as projected; returns [T, H, Dv]"""
    T, H = q.shape[:2]
    per = H // k.shape[1]
    freq, amp = rot_frequencies(rot)
    vfreq = plain_frequencies(v.shape[-1], float(rot["base"]))
    q, k, v = turn(q, positions, freq, amp), turn(k, positions, freq, amp), turn(v, positions, vfreq)
    s = torch.einsum("ihd,jhd->hij", q, k.repeat_interleave(per, 1)) * scale
    s = cap_scores(s, cap).masked_fill(~causal(T)[None], float("-inf"))
    o = torch.einsum("hij,jhd->ihd", softmax_with_one(s), v.repeat_interleave(per, 1))
    return turn(o, positions, vfreq, back=True)


def attention_mixer(h, W, m, eps):
    T = h.shape[0]
    H, G, D, Dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ W[n].T + W[n + ".b"] for n in ("q", "k", "v"))
    o = turned_value_attention(q.view(T, H, D), k.view(T, G, D), v.view(T, G, Dv), torch.arange(T), m["rot"], float(m["scale"]), float(m["softcap"]))
    return o.reshape(T, H * Dv) @ W["o"].T


def latent_attention_mixer(h, W, m, eps):
    T = h.shape[0]
    H, D, Dr, Dv, R = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    freq, amp = rot_frequencies(dict(m["rot"], dims=Dr))
    q = ((unit_rms(h @ W["dq"].T, eps) * W["dq.norm"]) @ W["uq"].T).view(T, H, D + Dr)
    down = h @ W["dkv"].T
    c = unit_rms(down[:, :R], eps) * W["dkv.norm"]
    shared = turn(down[:, None, R:], pos, freq, amp, interleaved=True)[:, 0]
    qr = turn(q[..., D:], pos, freq, amp, interleaved=True)
    k, v = (c @ W["uk"].T).view(T, H, D), (c @ W["uv"].T).view(T, H, Dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :D], k) + torch.einsum("ihd,jd->hij", qr, shared)) * float(m["scale"])
    p = torch.softmax(s.masked_fill(~causal(T)[None], float("-inf")), dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v).reshape(T, H * Dv) @ W["o"].T


def mlstm_gates(i_logit, f_logit, cap):
    """(log input gate, log forget gate)"""
    i = cap * torch.tanh(i_logit / cap)
    z = cap * torch.tanh(f_logit / cap)
    return i, torch.nn.functional.logsigmoid(z)


def mlstm_parts(q, k, v, i, f, state=None):
    """q (already scaled), k [T, H, D]; v [T, H, Dv]; i, f [T, H] log gates.  Returns (S^T q [T, H, Dv], denominators [T, H], (S, n, m))"""
    T, H, D = q.shape
    S, n, m = state if state is not None else (torch.zeros(H, D, v.shape[-1], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype))
    above, below = [], []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + take[:, None, None] * k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        n = keep[:, None] * n + take[:, None] * k[t]
        below.append(torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6)
        above.append(torch.einsum("hij,hi->hj", S, q[t]))
    return torch.stack(above), torch.stack(below), (S, n, m)


def mlstm_scan(q, k, v, i, f, state=None):
    """(outputs [T, H, Dv], (S, n, m))"""
    above, below, state = mlstm_parts(q, k, v, i, f, state)
    return above / below.unsqueeze(-1), state


def mlstm_mixer(h, W, m, eps):
    T = h.shape[0]
    H, D, Dv, cap = m["heads"], m["dim"], m["vdim"], float(m["gate_cap"])
    q, k, v = (h @ W["q"].T).view(T, H, D) * D ** -0.5, (h @ W["k"].T).view(T, H, D), (h @ W["v"].T).view(T, H, Dv)
    i, f = mlstm_gates(h @ W["i"].T + W["i.b"], h @ W["f"].T + W["f.b"], cap)
    o, _ = mlstm_scan(q, k, v, i, f)
    return (unit_rms(o, eps).reshape(T, H * Dv) * W["norm"] * torch.sigmoid(h @ W["g"].T)) @ W["o"].T


MIXERS = {"attention": attention_mixer, "latent_attention": latent_attention_mixer, "mlstm": mlstm_mixer}


def feed_forward(h, W):
    return (gelu_tanh(h @ W["gate"].T) * (h @ W["up"].T)) @ W["down"].T


# ------------------------------------------------------------------ the model
def layer_runs(cfg):
    """(layer, True where the embedding output is added first) in the order in which layers run"""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def enter_pass(x, x0):
    return x + x0


def forward(cfg, weights, tokens, collect=None):
    """logits [T, vocab] of one sequence; ``collect``: a list that receives the stream after every layer run"""
    eps = float(cfg["norm"]["eps"])
    x0 = x = weights["embed"][torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    for i, again in layer_runs(cfg):
        if again:
            x = enter_pass(x, x0)
        lc, W = cfg["layers"][i], sub(weights, f"l{i}.")
        y = MIXERS[lc["type"]](zero_centred_norm(x, W["norm1"], eps), sub(W, "mix."), lc["mixer"], eps)
        if lc.get("mlp") is not None:
            y = y + feed_forward(zero_centred_norm(x, W["norm2"], eps), sub(W, "mlp."))
        x = x + y
        if collect is not None:
            collect.append(x.clone())
    return zero_centred_norm(x, weights["final.norm"], eps) @ weights["head"].T


def greedy(cfg, weights, prompt, n_new):
    tokens = list(prompt)
    for _ in range(n_new):
        tokens.append(int(forward(cfg, weights, tokens)[-1].argmax()))
    return tokens


# ------------------------------------------------------------------ random models
ATT = dict(heads=6, kv_heads=2, dim=12, vdim=10, rot_dims=8, base=50.0, scale=0.5, softcap=4.0)
LAT = dict(heads=4, dim=10, rot_dim=6, vdim=14, kv_rank=18, q_rank=22, base=300.0, scale=0.4, scaling=dict(factor=3.0, original=64, fast=8.0, slow=1.0))
MEM = dict(heads=3, dim=10, vdim=14, gate_cap=6.0)


def random_config(width=40, vocab=61, order=("attention", "latent_attention", "mlstm", "attention"), ffs=(24, 56, None, 33), att=None, lat=None, mem=None,
                  loop=(1, 3, 3), eps=1e-5, embed_scale=2.5):
    """``order``: the layers' mixers; ``ffs``: per layer the feed-forward's width or None; the dicts override the sizes above;
    ``loop``: (start, stop, times) or None"""
    a, l, m = (dict(base, **(over or {})) for base, over in ((ATT, att), (LAT, lat), (MEM, mem)))
    rot_l = {"base": l["base"], "dims": l["rot_dim"]}
    if l["scaling"]:
        rot_l["scaling"] = dict(l["scaling"])
    mixers = {"attention": dict({k: a[k] for k in ("heads", "kv_heads", "dim", "vdim", "scale", "softcap")}, rot={"base": a["base"], "dims": a["rot_dims"]}),
              "latent_attention": dict({k: l[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale")}, rot=rot_l),
              "mlstm": dict(m)}
    layers = [{"type": kind, "mixer": mixers[kind], "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for kind, ff in zip(order, ffs)]
    cfg = {"architecture": "Rumuvik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale}, "layers": layers}
    if loop:
        cfg["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return cfg


def random_weights(cfg, seed, dtype=torch.bfloat16):
    """weights under the checkpoint's names"""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def mat(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def vec(n, mean=0.0, s=0.2):
        return mean + torch.randn(n, generator=g) * s

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g), "final.norm": vec(W), "head": mat(cfg["vocab"], W)}
    for i, lc in enumerate(cfg["layers"]):
        p, m = f"l{i}.", lc["mixer"]
        w[p + "norm1"] = vec(W)
        x = p + "mix."
        H, D, Dv = m["heads"], m["dim"], m["vdim"]
        if lc["type"] == "attention":
            G = m["kv_heads"]
            for n, rows in (("q", H * D), ("k", G * D), ("v", G * Dv)):
                w[x + n], w[x + n + ".b"] = mat(rows, W, 1.5), vec(rows, 0.0, 0.5)
        elif lc["type"] == "latent_attention":
            R, Dr, Q = m["kv_rank"], m["rot_dim"], m["q_rank"]
            w[x + "dq"], w[x + "dq.norm"], w[x + "uq"] = mat(Q, W), vec(Q, 1.0), mat(H * (D + Dr), Q, 1.5)
            w[x + "dkv"], w[x + "dkv.norm"] = mat(R + Dr, W, 1.5), vec(R, 1.0)
            w[x + "uk"], w[x + "uv"] = mat(H * D, R, 1.5), mat(H * Dv, R)
        else:
            for n, rows in (("q", H * D), ("k", H * D), ("v", H * Dv), ("g", H * Dv)):
                w[x + n] = mat(rows, W, 1.5)
            w[x + "i"], w[x + "f"] = mat(H, W, 2.0), mat(H, W, 1.5)
            w[x + "i.b"], w[x + "f.b"], w[x + "norm"] = vec(H, -0.5, 1.0), vec(H, 2.5, 1.0), vec(H * Dv, 1.0)
        w[x + "o"] = mat(W, H * Dv)
        if lc.get("mlp") is not None:
            F = lc["mlp"]["ff"]
            w[p + "norm2"], w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"] = vec(W), mat(F, W, 2.0), mat(F, W), mat(W, F)
    return {k: v.to(dtype) for k, v in w.items()}
