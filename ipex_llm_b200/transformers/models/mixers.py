"""Pieces that several of this package's own designs are built from: the rotary frequencies of a ``rot`` block, a lone weight under
a module of its own, short convolutions on a layer's state, and the **delta rule with a decay per key channel** (behind short
convolutions, unit-norm q / k, a per-head RMS norm of the read-out and a low-rank sigmoid gate) with its module tree, and the
attention over a **latent cache** whose rows hold a normalised latent and one rotated key part that all heads share.  The kernels
are those of ``mixer_ops``."""
import math

import torch
from torch import nn

from ipex_llm_b200.transformers.models import mixer_ops as ops
from ipex_llm_b200.utils.common import invalidInputError

ABSORB_MAX_TOKENS = 16        # up to this many new tokens per row attend to a latent cache itself (no key / value expansion)
YARN_AMP_SLOPE = 0.1          # cosine and sine of rescaled frequencies are multiplied by slope * ln(factor) + 1


def rotary_frequencies(rot):
    """(frequency of every rotated pair as a list of floats, amplitude) of a ``rot`` block: base^(-2i / dims); with ``scaling``
    (factor, original, fast, slow) a pair whose wavelength makes fewer than ``slow`` turns within ``original`` positions is slowed
    down by ``factor``, one that makes more than ``fast`` turns is kept, the pairs between are blended linearly by their index,
    and cosine and sine are multiplied by 0.1 ln(factor) + 1"""
    dims, base = int(rot["dims"]), float(rot["base"])
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair_with_turns(turns):                              # the (fractional) pair index whose wavelength makes this many turns
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(pair_with_turns(float(sc["fast"]))), 0)
    hi = min(math.ceil(pair_with_turns(float(sc["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, YARN_AMP_SLOPE * math.log(factor) + 1.0


class Rotary:
    """frequencies of a ``rot`` block in double precision on the device they are needed on (not a buffer: ``model.to(dtype)`` must
    not round them; the kernel forms the angles in double precision too)"""

    def __init__(self, rot):
        self.dims = int(rot["dims"])
        invalidInputError(self.dims % 2 == 0, "rotary dims must be even")
        self.freq, self.amp = rotary_frequencies(rot)
        self._on = {}

    def inv_freq(self, device):
        t = self._on.get(device)
        if t is None:
            t = self._on[device] = torch.tensor(self.freq or [0.0], dtype=torch.float64).to(device)
        return t


class Angles:
    """cosine and sine of every new token and rotated pair, formed once per call for all layer runs that share the frequencies"""

    def __init__(self, B, S, cache, dyn):
        self.B, self.S, self.cache, self.dyn = B, S, cache, dyn
        self._tables = {}

    def of(self, rotary, device):
        """fp32 [B * S, pairs, 2], or None where nothing is rotated"""
        if not rotary.freq:
            return None
        key = (tuple(rotary.freq), rotary.amp)
        t = self._tables.get(key)
        if t is None:                                        # position = slot - padding; a recorded step reads its slot from the device
            t = self._tables[key] = ops.rotary_table(rotary.inv_freq(device), rotary.amp, self.B, self.S, self.cache.seen, 0, self.cache.pad, dyn=self.dyn)
        return t


def latent_expansion(uk, uv, heads, dim, rot_dim, vdim, rank):
    """[heads * (dim + rot_dim) + heads * vdim, rank + rot_dim] from per-head key rows uk [heads * dim, rank] and value rows uv
    [heads * vdim, rank]: turns cache rows [latent | rotated key part] into every head's key [W_uk latent | rotated part] and value
    W_uv latent; per head the key rows are (W_uk_h 0; 0 I), the value rows (W_uv_h 0)"""
    keys = torch.zeros(heads, dim + rot_dim, rank + rot_dim, dtype=uk.dtype)
    keys[:, :dim, :rank] = uk.view(heads, dim, rank)
    keys[:, dim:, rank:] = torch.eye(rot_dim, dtype=uk.dtype)
    values = torch.zeros(heads * vdim, rank + rot_dim, dtype=uk.dtype)
    values[:, :rank] = uv
    return torch.cat([keys.view(heads * (dim + rot_dim), rank + rot_dim), values], dim=0)


def latent_cache_attention(q, w, store, B, S, heads, q_dim, vdim, rank, held, shift, pad, scale, out, window=0, dyn=None, tensor_cores=True):
    """out[:, : heads * vdim] = softmax attention of the new tokens' queries q [B * S, heads * q_dim] over the cache rows ``store`` [B,
    capacity, rank + rotated part]; ``w``: ``latent_expansion``.

    Few new tokens move their queries into the cache rows' space (W_uk_h^T q | rotated q): the cache itself is then the key of one
    shared head, its latent part the value, and W_uv_h maps the weighted latents back.  A prompt or a long portion expands the keys
    and values of the positions that some new token still sees."""
    H, N, row = heads, B * S, store.shape[2]
    if S <= ABSORB_MAX_TOKENS:
        wk, wv = w[:H * q_dim].view(H, q_dim, row), w[H * q_dim:].view(H, vdim, row)[:, :, :rank]
        qa = torch.matmul(q.view(N, H, q_dim).transpose(0, 1), wk).transpose(0, 1)                  # [N, H, row], stored head by head
        rows = store.unsqueeze(2)                                            # [B, capacity, 1, row]
        o_rows = ops.softmax_attention(qa, rows, rows[..., :rank], B, S, H, held, shift, pad, window, scale, dyn=dyn)
        o = torch.matmul(o_rows.view(N, H, rank).transpose(0, 1), wv.transpose(1, 2))               # [H, N, vdim]
        out[:, :H * vdim].unflatten(1, (H, vdim)).copy_(o.transpose(0, 1))
        return
    first = max(held - (window - 1), 0) if window > 0 else 0
    total = held + S
    kvx = torch.nn.functional.linear(store[:, first:total], w)               # [B, total - first, H * (q_dim + vdim)]
    k, v = kvx[..., :H * q_dim].view(B, total - first, H, q_dim), kvx[..., H * q_dim:].view(B, total - first, H, vdim)
    ops.softmax_attention(q, k, v, B, S, H, held - first, shift + first, pad, window, scale, out=out, tensor_cores=tensor_cores)


class Weight(nn.Module):
    """a lone parameter under the name ``<module>.weight``: a norm's vector of weights, or (shape ()) its single gain"""

    def __init__(self, *shape):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(tuple(shape)))


class ChannelDeltaMixer(nn.Module):
    """``PARTS`` are the projections that read the mixer's input: a design merges them, in this order, into one ``in_proj``"""
    PARTS = ("q_proj", "k_proj", "v_proj", "b_proj", "a1_proj", "g1_proj")

    def __init__(self, width, m, ranks):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim, self.taps = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"])
        invalidInputError(self.kv_heads >= 1 and self.heads % self.kv_heads == 0, "heads must be a multiple of kv_heads")
        qk, v = self.kv_heads * self.dim, self.heads * self.vdim
        self.q_proj, self.k_proj, self.v_proj = nn.Linear(width, qk, bias=False), nn.Linear(width, qk, bias=False), nn.Linear(width, v, bias=False)
        self.b_proj = nn.Linear(width, self.heads, bias=False)
        self.a1_proj, self.a2_proj = nn.Linear(width, ranks[0], bias=False), nn.Linear(ranks[0], self.heads * self.dim, bias=False)
        self.g1_proj, self.g2_proj = nn.Linear(width, ranks[1], bias=False), nn.Linear(ranks[1], v, bias=False)
        self.conv_weight = nn.Parameter(torch.zeros(2 * qk + v, self.taps))          # q | k | v channels
        self.A_log, self.dt_bias = nn.Parameter(torch.zeros(self.heads)), nn.Parameter(torch.zeros(self.heads * self.dim))
        self.norm = Weight(self.vdim)
        self.o_proj = nn.Linear(v, width, bias=False)



    @property
    def conv_channels(self):
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def in_columns(self):
        """columns of the merged input projection: q | k | v | beta | decay rank | gate rank"""
        return self.conv_channels + self.heads + self.a2_proj.in_features + self.g2_proj.in_features


def short_conv(proj, off, channels, weight, bias, rec, key, B, S, cache, silu, add_input=False):
    """a short causal convolution over the new tokens and the state's tail (which keeps its address: a recorded step holds it)"""
    taps = weight.shape[1]
    tail, tail_next = rec.tails(B, taps, channels, proj.dtype, proj.device, key=key)
    pad = cache.pad if cache.seen == 0 else None                             # padding only ever precedes a row's first call
    y = ops.short_conv(proj, off, channels, weight, bias, tail, tail if S == 1 else tail_next, cache.seen, pad, silu=silu, add_input=add_input)
    if S > 1:
        tail.copy_(tail_next)
    return y


def channel_delta(mx, proj, off, rec, B, S, cache, eps, out, out_col=0, scale=1.0):
    """the delta rule over the new tokens: ``proj`` [N, P] holds the merged input projection from column ``off`` on; writes
    ``scale`` * (normed, gated read-out) into out[:, out_col : out_col + heads * vdim]"""
    H, G, D, Dv, P = mx.heads, mx.kv_heads, mx.dim, mx.vdim, proj.shape[1]
    off_b = off + mx.conv_channels
    off_a1 = off_b + H
    off_g1 = off_a1 + mx.a2_proj.in_features
    proj3 = proj.view(B, S, P)
    conv = short_conv(proj3, off, mx.conv_channels, mx.conv_weight, None, rec, "mixer", B, S, cache, silu=True)
    z = mx.a2_proj(proj[:, off_a1:off_g1])                                   # decay logits [N, H D]
    gate = mx.g2_proj(proj[:, off_g1:off_g1 + mx.g2_proj.in_features])       # [N, H Dv]
    state = rec.matrix(B, H, D, Dv, proj.device)
    o = ops.channel_delta_rule(conv, G, H, D, Dv, proj3, off_b, z, mx.A_log, mx.dt_bias, state, cache.seen, cache.pad if cache.seen == 0 else None)
    ops.gated_rms_norm(o, gate, 0, mx.norm.weight, eps, out, out_col, scale, sigmoid=True)


class Constants:
    """numbers of a configuration as a vector on the device and in the type they are needed in (not a buffer: ``model.to(dtype)``
    must not round them)"""

    def __init__(self, values):
        self.values = [float(v) for v in values]
        self._on = {}

    def on(self, device, dtype=torch.float32):
        t = self._on.get((device, dtype))
        if t is None:
            t = self._on[(device, dtype)] = torch.tensor(self.values, dtype=torch.float64).to(dtype).to(device)
        return t


def linear_f32(linear, x):
    """a bias-free projection whose 32-bit accumulator is the result (a plain 16-bit linear; a converted one answers in its own type)"""
    if type(linear) is nn.Linear and x.dtype in (torch.bfloat16, torch.float16) and x.device.type == "cuda":
        return torch.mm(x, linear.weight.t(), out_dtype=torch.float32)
    return linear(x)


def plain_linears(model):
    """no projection was converted to a low-bit format (those products share one workspace per device, so two of them must not run on
    two streams at once)"""
    plain = model.__dict__.get("_b200_plain_linears")
    if plain is None:
        plain = model.__dict__["_b200_plain_linears"] = all(type(m) is nn.Linear for m in model.modules() if isinstance(m, nn.Linear) or
                                                            type(m).__name__ == "LowBitLinear")
    return plain
