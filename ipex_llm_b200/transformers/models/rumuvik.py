"""Rumuvik: a decoder-only design whose layers run their mixer and their feed-forward side by side on the same stream,

    x <- x + (mixer(norm1(x)) + ff(norm2(x))),

with RMS norms whose weights are stored around zero (x / rms(x) * (1 + w)) and a stretch of layers that runs several times in a row
with the same weights: in front of every pass but the first the embedding output is added to the stream, and every pass keeps a cache
or state of its own.  A layer's mixer is one of

* ``attention``: grouped softmax attention with biases in its projections, capped scores and a one in the softmax's denominator (a
  sink of score 0 that has no value), whose **values are rotated** by their own position over all their channels; every head's
  output is turned back by the query's position;
* ``latent_attention``: softmax attention whose queries go through a normalised latent of their own and whose keys and values are
  expanded per head from one normalised latent per position, plus one rotated key part that all heads share (latent and rotated part
  are all the cache keeps); rotary frequencies may be rescaled between a fast and a slow band, pairs are neighbouring channels;
* ``mlstm``: the matrix memory of an xLSTM: exponential input gate and sigmoid forget gate from capped logits, a running maximum that
  keeps both in range, a normaliser, a per-head RMS norm of the read-out and a sigmoid gate per channel;

and its feed-forward (optional) is ``down(gelu_tanh(gate h) * up h)``.  The embedding is multiplied by a constant of the configuration.

No library ships this model.  The module tree, the configuration reader and the checkpoint's name map live here; the state in
``transformers/kv.py`` (``DynamicStateCache``: one key/value store, latent cache or matrix state per layer RUN), the kernels in
``csrc/mixers`` behind ``ggml/model/mixers_cpp.py``.  The projections are ``nn.Linear`` modules, so the low-bit conversion treats
them like any other model's.  The residual stream, every norm, rotary angles, attention scores and weights and everything inside the
recurrence are 32-bit whatever the model's dtype.
"""
import json
import os
from typing import Optional

import torch
from torch import nn
from transformers import GenerationMixin, PreTrainedConfig, PreTrainedModel
from transformers.modeling_outputs import CausalLMOutputWithPast

from ipex_llm_b200.transformers.kv import DynamicStateCache
from ipex_llm_b200.transformers.models import mixer_ops as ops
from ipex_llm_b200.transformers.models.common import merge_linear, merge_linear_inputs, zero_rows
from ipex_llm_b200.transformers.models.mixers import (Angles, Constants, Rotary, Weight, latent_cache_attention, latent_expansion, linear_f32,
                                                      plain_linears)
from ipex_llm_b200.transformers.models.utils import read_safetensors
from ipex_llm_b200.utils.common import invalidInputError

OVERLAP_MIN_TOKENS = 256      # from this many new tokens on, a layer's feed-forward runs on a second stream beside its mixer
MLSTM_TINY = 1e-6             # added to the mLSTM's denominator


class RumuvikConfig(PreTrainedConfig):
    """config.json of the design: ``vocab``, ``width``, ``layers`` (per layer: ``type``, ``mixer`` sizes and constants, ``mlp`` or
    null), ``loop`` (``start``, ``stop``, ``times``; optional), ``norm.eps``, ``embedding.scale``"""
    model_type = "rumuvik"

    def __init__(self, vocab=256, width=64, layers=None, loop=None, norm=None, embedding=None, architecture="Rumuvik", **kwargs):
        self.vocab, self.width = int(vocab), int(width)
        self.layers = layers or []
        self.loop = loop
        self.norm = norm or {"eps": 1e-5}
        self.embedding = embedding or {"scale": 1.0}
        self.architecture = architecture
        kwargs["tie_word_embeddings"] = False
        super().__init__(**kwargs)
        self.vocab_size, self.hidden_size, self.num_hidden_layers = self.vocab, self.width, len(self.layers)
        self.use_cache = True

    @property
    def norm_eps(self):
        return float(self.norm["eps"])

    @property
    def embedding_scale(self):
        return float(self.embedding.get("scale", 1.0))

    def layer_runs(self):
        """[(layer, again)]: the layers in the order in which they run; ``again``: a pass but the first starts with this run (the
        embedding output is added in front of it)"""
        n = len(self.layers)
        times = int(self.loop.get("times", 1)) if self.loop else 1
        if times == 1:
            return [(i, False) for i in range(n)]
        start, stop = int(self.loop["start"]), int(self.loop["stop"])
        invalidInputError(0 <= start < stop <= n and times >= 1, "loop: start .. stop - 1 must name layers that run at least once")
        looped = [(i, t > 0 and i == start) for t in range(times) for i in range(start, stop)]
        return [(i, False) for i in range(start)] + looped + [(i, False) for i in range(stop, n)]


class TurnedValueAttention(nn.Module):
    """``q_proj`` / ``k_proj`` / ``v_proj`` become one ``in_proj`` when ``merge_projections`` has run"""
    PARTS = ("q_proj", "k_proj", "v_proj")

    def __init__(self, width, m):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
        invalidInputError(self.kv_heads >= 1 and self.heads % self.kv_heads == 0, "heads must be a multiple of kv_heads")
        self.scale, self.softcap = float(m["scale"]), float(m.get("softcap") or 0.0)
        self.rotary = Rotary(m["rot"])
        invalidInputError(self.rotary.dims <= self.dim, "rotary dims exceed the head size")
        self.value_rotary = Rotary({"dims": self.vdim, "base": m["rot"]["base"]})       # all channels, never rescaled
        self.sink = Constants([0.0] * self.heads)             # the score of the one in the softmax's denominator
        self.q_proj = nn.Linear(width, self.heads * self.dim, bias=True)
        self.k_proj = nn.Linear(width, self.kv_heads * self.dim, bias=True)
        self.v_proj = nn.Linear(width, self.kv_heads * self.vdim, bias=True)
        self.o_proj = nn.Linear(self.heads * self.vdim, width, bias=False)


class QueryLatentAttention(nn.Module):
    """``dq`` and ``dkv`` become one ``in_proj`` when ``merge_projections`` has run.  A cache row is [latent | rotated key part];
    ``expand``: see ``latent_expansion`` (a plain parameter: the attention of few tokens multiplies by its per-head blocks)"""
    PARTS = ("dq", "dkv")

    def __init__(self, width, m):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.kv_rank, self.q_rank = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank",
                                                                                                    "q_rank"))
        self.scale = float(m["scale"])
        self.rotary = Rotary(dict(m["rot"], dims=self.rot_dim))
        qd = self.dim + self.rot_dim
        self.dq, self.dq_norm = nn.Linear(width, self.q_rank, bias=False), Weight(self.q_rank)
        self.uq = nn.Linear(self.q_rank, self.heads * qd, bias=False)
        self.dkv, self.dkv_norm = nn.Linear(width, self.kv_rank + self.rot_dim, bias=False), Weight(self.kv_rank)
        self.expand = Weight(self.heads * (qd + self.vdim), self.kv_rank + self.rot_dim)
        self.o_proj = nn.Linear(self.heads * self.vdim, width, bias=False)


class MatrixMemory(nn.Module):
    """the mLSTM; the six projections of the input become one ``in_proj`` when ``merge_projections`` has run (the gates' biases stay
    apart: they are added in 32-bit where the gates are formed)"""
    PARTS = ("q_proj", "k_proj", "v_proj", "g_proj", "i_proj", "f_proj")

    def __init__(self, width, m):
        super().__init__()
        self.heads, self.dim, self.vdim, self.cap = int(m["heads"]), int(m["dim"]), int(m["vdim"]), float(m["gate_cap"])
        qk, v = self.heads * self.dim, self.heads * self.vdim
        self.q_proj, self.k_proj = nn.Linear(width, qk, bias=False), nn.Linear(width, qk, bias=False)
        self.v_proj, self.g_proj = nn.Linear(width, v, bias=False), nn.Linear(width, v, bias=False)
        self.i_proj, self.f_proj = nn.Linear(width, self.heads, bias=False), nn.Linear(width, self.heads, bias=False)
        self.i_bias, self.f_bias = nn.Parameter(torch.zeros(self.heads)), nn.Parameter(torch.zeros(self.heads))
        self.norm = Weight(v)
        self.o_proj = nn.Linear(v, width, bias=False)


class GatedMLP(nn.Module):
    """down(gelu_tanh(gate h) * up h), no biases; gate and up are the two halves of ``gate_up``'s rows"""

    def __init__(self, width, m):
        super().__init__()
        invalidInputError(m.get("kind", "dense") == "dense", f"unknown feed-forward kind {m.get('kind')}")
        self.ff = int(m["ff"])
        self.gate_up, self.down_proj = nn.Linear(width, 2 * self.ff, bias=False), nn.Linear(self.ff, width, bias=False)


MIXERS = {"attention": TurnedValueAttention, "latent_attention": QueryLatentAttention, "mlstm": MatrixMemory}


class RumuvikLayer(nn.Module):
    """``out_proj`` (mixer output and feed-forward: their sum is taken in the accumulator of one product over [mixer's heads |
    activations]) appears when ``merge_projections`` has run"""

    def __init__(self, config: RumuvikConfig, index):
        super().__init__()
        lc, w = config.layers[index], config.width
        self.kind = lc["type"]
        invalidInputError(self.kind in MIXERS, f"unknown layer type {self.kind}")
        self.norm1 = Weight(w)
        self.mixer = MIXERS[self.kind](w, lc["mixer"])
        self.mlp = None
        if lc.get("mlp") is not None:
            self.norm2 = Weight(w)
            self.mlp = GatedMLP(w, lc["mlp"])

    @property
    def mixed_columns(self):
        return self.mixer.heads * self.mixer.vdim


def merge_projections(module: nn.Module, row_multiple: int = 0):
    """every projection that reads a mixer's input becomes one ``in_proj``, a layer's two output projections one ``out_proj``;
    ``row_multiple``: see ``zero_rows`` (the kernels address columns by offset, the extra ones are never read)"""
    if not isinstance(module, RumuvikLayer) or hasattr(module, "out_proj"):
        return
    mx = module.mixer
    parts = [getattr(mx, n) for n in mx.PARTS]
    mx.in_proj = merge_linear(parts + zero_rows(parts[0], sum(p.weight.shape[0] for p in parts), row_multiple))
    for n in mx.PARTS:
        delattr(mx, n)
    module.out_proj = merge_linear_inputs([mx.o_proj] + ([module.mlp.down_proj] if module.mlp is not None else []))
    del mx.o_proj
    if module.mlp is not None:
        del module.mlp.down_proj


class RumuvikModel(nn.Module):
    def __init__(self, config: RumuvikConfig):
        super().__init__()
        self.config = config
        self.embed_tokens = nn.Embedding(config.vocab, config.width)
        self.layers = nn.ModuleList([RumuvikLayer(config, i) for i in range(len(config.layers))])
        self.norm = Weight(config.width)


class RumuvikForCausalLM(PreTrainedModel, GenerationMixin):
    config_class = RumuvikConfig
    base_model_prefix = "model"
    _no_split_modules = ["RumuvikLayer"]
    _supports_attention_backend = False
    main_input_name = "input_ids"

    def __init__(self, config: RumuvikConfig):
        super().__init__(config)
        self.model = RumuvikModel(config)
        self.lm_head = nn.Linear(config.width, config.vocab, bias=False)
        self.collect_residual = None          # a list: gets the residual stream after every layer run (debugging aid)
        self.attention_tensor_cores = True    # 16-bit models: prompts take the tensor-core attention kernel
        self.overlap_feed_forward = True      # mixer and feed-forward read the same stream, so they run side by side
        self._side_stream = None

    def _init_weights(self, module):
        pass

    def get_input_embeddings(self):
        return self.model.embed_tokens

    def get_output_embeddings(self):
        return self.lm_head

    # ---- mixers (h: the mixer's input in the model's dtype, [N, W]); each writes its heads into the first columns of ``out``
    def _attention(self, mx, h, out, st, B, S, cache, angles):
        H, G, D, Dv = mx.heads, mx.kv_heads, mx.dim, mx.vdim
        proj = mx.in_proj(h)                                                 # q | k | v
        kv = st.kv
        like_k, like_v = (torch.empty((B, G, 0, d), dtype=h.dtype, device=h.device) for d in (D, Dv))
        k_store, v_store, held = kv.slots(like_k, like_v, S)
        shift = cache.seen - held                                            # storage index + shift = slot number
        # a recorded decode step reads the length from the device (the value given here is the one at recording time)
        dyn = kv.length_dev if (cache.frozen and S == 1) else None
        cap = kv.capacity()
        table, turned = angles.of(mx.rotary, h.device), angles.of(mx.value_rotary, h.device)
        q = ops.rope_qk_prepare(proj.view(B, S, -1), 0, H * D, (H + G) * D, H, G, D, D, Dv, 0, 0, mx.rotary.dims, None, 1.0, k_store,
                                (G * cap * D, D, cap * D), v_store, (G * cap * Dv, Dv, cap * Dv), held, shift, cache.pad, dyn=dyn, table=table,
                                v_table=turned)
        kv.commit(S)
        ops.softmax_attention(q, k_store.permute(0, 2, 1, 3), v_store.permute(0, 2, 1, 3), B, S, H, held, shift, cache.pad, 0, mx.scale, out=out,
                              dyn=dyn, tensor_cores=self.attention_tensor_cores, softcap=mx.softcap, sink=mx.sink.on(h.device, h.dtype), back=turned)

    def _latent_attention(self, mx, h, out, st, B, S, cache, angles):
        H, D, Dr, R, eps = mx.heads, mx.dim, mx.rot_dim, mx.kv_rank, self.config.norm_eps
        kv = st.kv
        proj = mx.in_proj(h).view(B, S, -1)                                  # query latent | latent | rotated key part
        store, held = kv.slots(B, R + Dr, S, h.dtype, h.device)
        shift = cache.seen - held
        dyn = kv.length_dev if (cache.frozen and S == 1) else None
        cap = store.shape[1]
        q = mx.uq(ops.rms_norm_columns(proj, 0, mx.q_rank, mx.dq_norm.weight, eps, held, shift, cache.pad, dyn=dyn))
        q = ops.rope_qk_prepare(q.view(B, S, -1), 0, mx.q_rank, 0, H, 1, D + Dr, R + Dr, 0, D, R, Dr, None, 1.0, store, (cap * (R + Dr), R + Dr, 0), None,
                                None, held, shift, cache.pad, eps=eps, k_norm_w=mx.dkv_norm.weight, k_norm_cols=R, dyn=dyn,
                                table=angles.of(mx.rotary, h.device), interleaved=True, kv_proj=proj)
        kv.commit(S)
        latent_cache_attention(q, mx.expand.weight, store, B, S, H, D + Dr, mx.vdim, R, held, shift, cache.pad, mx.scale, out, dyn=dyn,
                               tensor_cores=self.attention_tensor_cores)

    def _mlstm(self, mx, h, out, st, B, S, cache):
        H, D, Dv = mx.heads, mx.dim, mx.vdim
        proj = mx.in_proj(h)                                                 # q | k | v | gate | input gate | forget gate
        off_k, off_v = H * D, 2 * H * D
        off_g, off_i = off_v + H * Dv, off_v + 2 * H * Dv
        rec, dev = st.rec, h.device
        o, below = ops.mlstm(proj.view(B, S, -1), 0, off_k, off_v, off_i, off_i + H, H, D, Dv, mx.i_bias, mx.f_bias, mx.cap, MLSTM_TINY,
                             rec.matrix(B, H, D, Dv, dev), rec.vector("normaliser", (B, H, D), dev), rec.vector("maximum", (B, H, Dv + 1), dev),
                             cache.seen, cache.pad if cache.seen == 0 else None)
        ops.gated_rms_norm(o, proj, off_g, mx.norm.weight, self.config.norm_eps, out, 0, 1.0, sigmoid=True, below=below)

    def _mix(self, layer, h, out, st, B, S, cache, angles):
        if layer.kind == "attention":
            self._attention(layer.mixer, h, out, st, B, S, cache, angles)
        elif layer.kind == "latent_attention":
            self._latent_attention(layer.mixer, h, out, st, B, S, cache, angles)
        else:
            self._mlstm(layer.mixer, h, out, st, B, S, cache)

    def _side(self, dev, tokens, recorded):
        """the stream on which feed-forwards run beside mixers, or None: prompts, and the step that is recorded (its launches overlap
        when it is replayed)"""
        if not (self.overlap_feed_forward and dev.type == "cuda" and plain_linears(self)):
            return None
        if not recorded and (tokens < OVERLAP_MIN_TOKENS or torch.cuda.is_current_stream_capturing()):
            return None
        if self._side_stream is None or self._side_stream.device != dev:
            self._side_stream = torch.cuda.Stream(dev)
        return self._side_stream

    def _layer(self, layer, h1, h2, st, B, S, cache, angles, side):
        """[N, W]: mixer(h1) + ff(h2)"""
        invalidInputError(hasattr(layer, "out_proj"), "the projections are merged at load time (merge_projections)")
        cols, mlp = layer.mixed_columns, layer.mlp
        out = torch.empty(B * S, cols + (mlp.ff if mlp is not None else 0), dtype=h1.dtype, device=h1.device)
        if mlp is None:
            self._mix(layer, h1, out, st, B, S, cache, angles)
            return linear_f32(layer.out_proj, out)
        if side is None:
            self._mix(layer, h1, out, st, B, S, cache, angles)
            ops.gelu_tanh_mul(mlp.gate_up(h2), mlp.ff, out=out[:, cols:])
            return linear_f32(layer.out_proj, out)
        # both halves write their columns of one buffer: everything that crosses the streams was allocated on the main one and
        # outlives the join
        main = torch.cuda.current_stream(h1.device)
        forked = main.record_event()
        self._mix(layer, h1, out, st, B, S, cache, angles)
        side.wait_event(forked)
        with torch.cuda.stream(side):
            ops.gelu_tanh_mul(mlp.gate_up(h2), mlp.ff, out=out[:, cols:])
        main.wait_stream(side)
        return linear_f32(layer.out_proj, out)

    def forward(self, input_ids: Optional[torch.LongTensor] = None, attention_mask: Optional[torch.Tensor] = None,
                position_ids=None, past_key_values=None, inputs_embeds=None, use_cache: Optional[bool] = None,
                logits_to_keep=0, **kwargs):
        """``input_ids`` [B, S]: the next S tokens of every row.  On the first call of a batch ``attention_mask`` [B, S] gives
        the left padding; later calls continue from ``past_key_values`` (a ``DynamicStateCache``; any other or no cache
        starts a new one).  Positions follow from the padding, ``position_ids`` is not read.  ``logits_to_keep``: 0 = all
        positions, n = the last n, or a 1-D tensor of positions."""
        invalidInputError(input_ids is not None and inputs_embeds is None, "the model takes token ids")
        core, cfg = self.model, self.config
        B, S = input_ids.shape
        W, eps = cfg.width, cfg.norm_eps
        dev, dtype = core.embed_tokens.weight.device, core.embed_tokens.weight.dtype
        cache = past_key_values
        if not isinstance(cache, DynamicStateCache):
            invalidInputError(cache is None or cache.get_seq_length() == 0, "a filled cache of another class cannot be continued")
            cache = DynamicStateCache()
        if cache.seen == 0:                                                  # a batch's first call: the mask gives the padding
            cache.start(attention_mask, B, S, dev)
        invalidInputError(cache.pad.shape[0] == B, "batch size differs from the cache's")
        input_ids = input_ids.to(dev).contiguous()
        runs = cfg.layer_runs()
        recorded = cache.frozen and S == 1
        side = self._side(dev, B * S, recorded)
        lengths = [l.kv.length_dev for l in cache.layers if l is not None and l.kv is not None] if recorded else []
        angles = Angles(B, S, cache, lengths[0] if lengths else None)        # every store of a recorded step holds the same positions
        # padding only occurs in a batch's first call; later calls (a replayed step among them, whose slot number is the one at
        # recording time) say so by passing no padding
        x0 = torch.empty(B * S, W, dtype=torch.float32, device=dev) if any(again for _, again in runs) else None
        x, _ = ops.embed_pair(core.embed_tokens.weight, cfg.embedding_scale, None, 0, 0, 0, input_ids, None, cache.seen,
                              cache.pad if cache.seen == 0 else None, dtype, x_copy=x0)
        # the last norm rides along with the last residual update when every position's logits are wanted
        keep_all = S == 1 or (isinstance(logits_to_keep, int) and logits_to_keep == 0)

        def hand_on(ys, run):
            """x += ys in front of layer run number ``run`` (and the embedding output, where a further pass starts); returns the two
            normalised streams that this run's mixer and feed-forward read"""
            if run == len(runs):
                return ops.sum_residual_norms(x, ys, dtype, eps, gain1=core.norm.weight if keep_all else None, gain_add=1.0)
            li, again = runs[run]
            layer = core.layers[li]
            return ops.sum_residual_norms(x, ys + ([x0] if again else []), dtype, eps, gain1=layer.norm1.weight,
                                          gain2=layer.norm2.weight if layer.mlp is not None else None, gain_add=1.0)

        h1, h2 = hand_on([], 0)
        for run, (li, _) in enumerate(runs):
            layer = core.layers[li]
            st = cache.run_state(run, window=0 if layer.kind == "attention" else None, latent=layer.kind == "latent_attention")
            y = self._layer(layer, h1, h2, st, B, S, cache, angles, side)
            if self.collect_residual is not None:
                self.collect_residual.append((x + y).view(B, S, -1))
            h1, h2 = hand_on([y], run + 1)
        cache.advance(S)
        if keep_all:
            hn = h1.view(B, S, W)
        else:
            idx = slice(-logits_to_keep, None) if isinstance(logits_to_keep, int) else logits_to_keep.to(dev)
            hn = ops.rms_norm_rows(x.view(B, S, W)[:, idx, :].contiguous(), None, core.norm.weight, eps, dtype, vec_add=1.0)
        # every kept position as a row of its own ([rows, 1, W]): a converted lm_head keeps only the last position of a long
        # sequence axis (the reference's prefill shortcut), and which positions to keep is decided here, by logits_to_keep
        logits = self.lm_head(hn.reshape(-1, 1, W)).to(torch.float32).view(B, hn.shape[1], -1)
        return CausalLMOutputWithPast(logits=logits, past_key_values=cache)

    def prepare_inputs_for_generation(self, input_ids, past_key_values=None, attention_mask=None, **kwargs):
        """generate() hands over every token so far; the model takes those its cache has not seen"""
        seen = past_key_values.get_seq_length() if isinstance(past_key_values, DynamicStateCache) else 0
        return {"input_ids": input_ids[:, seen:], "attention_mask": attention_mask, "past_key_values": past_key_values,
                "use_cache": True, "logits_to_keep": 1}


# ------------------------------------------------------------------ checkpoint
def checkpoint_key_map(config: RumuvikConfig):
    """the model's parameter names -> the checkpoint's tensor names: one name, or a list of them (concatenated by rows).  The latent
    attention's ``expand`` is not in the map: ``load_pretrained`` builds it from the key and value expansions."""
    m = {"model.embed_tokens.weight": "embed", "lm_head.weight": "head", "model.norm.weight": "final.norm"}
    for i, lc in enumerate(config.layers):
        d, s = f"model.layers.{i}.", f"l{i}."
        m[d + "norm1.weight"] = s + "norm1"
        dm, sm = d + "mixer.", s + "mix."
        m[dm + "o_proj.weight"] = sm + "o"
        if lc["type"] == "attention":
            for n in ("q", "k", "v"):
                m[dm + n + "_proj.weight"], m[dm + n + "_proj.bias"] = sm + n, sm + n + ".b"
        elif lc["type"] == "latent_attention":
            for n in ("dq", "uq", "dkv"):
                m[dm + n + ".weight"] = sm + n
            m[dm + "dq_norm.weight"], m[dm + "dkv_norm.weight"] = sm + "dq.norm", sm + "dkv.norm"
        else:
            for n in ("q", "k", "v", "g", "i", "f"):
                m[dm + n + "_proj.weight"] = sm + n
            m[dm + "i_bias"], m[dm + "f_bias"], m[dm + "norm.weight"] = sm + "i.b", sm + "f.b", sm + "norm"
        if lc.get("mlp") is not None:
            m[d + "norm2.weight"] = s + "norm2"
            m[d + "mlp.gate_up.weight"], m[d + "mlp.down_proj.weight"] = [s + "mlp.gate", s + "mlp.up"], s + "mlp.down"
    return m


def load_pretrained(model_dir, torch_dtype=None, device=None):
    """config.json + model.safetensors of the design -> a ``RumuvikForCausalLM``"""
    with open(os.path.join(model_dir, "config.json")) as f:
        config = RumuvikConfig(**json.load(f))
    tensors = read_safetensors(os.path.join(model_dir, "model.safetensors"))
    if torch_dtype in (None, "auto"):
        torch_dtype = tensors["embed"].dtype
    with torch.device("meta"):
        model = RumuvikForCausalLM(config)
    state = {}
    for dst, src in checkpoint_key_map(config).items():
        names = [src] if isinstance(src, str) else list(src)
        missing = [s for s in names if s not in tensors]
        invalidInputError(not missing, f"the checkpoint has no tensor {missing}")
        t = tensors[src] if isinstance(src, str) else torch.cat([tensors[s] for s in src], dim=0)
        state[dst] = t.to(torch_dtype)
    for i, layer in enumerate(model.model.layers):
        if layer.kind == "latent_attention":
            uk, uv, mx = f"l{i}.mix.uk", f"l{i}.mix.uv", layer.mixer
            invalidInputError(uk in tensors and uv in tensors, f"the checkpoint has no tensor {[n for n in (uk, uv) if n not in tensors]}")
            invalidInputError(tuple(tensors[uk].shape) == (mx.heads * mx.dim, mx.kv_rank) and tuple(tensors[uv].shape) == (mx.heads * mx.vdim, mx.kv_rank),
                              f"l{i}: the key / value expansions do not have the sizes the configuration gives")
            state[f"model.layers.{i}.mixer.expand.weight"] = latent_expansion(tensors[uk].to(torch_dtype), tensors[uv].to(torch_dtype), mx.heads, mx.dim,
                                                                              mx.rot_dim, mx.vdim, mx.kv_rank)
    for name, p in model.named_parameters():
        invalidInputError(name in state, f"no checkpoint tensor for parameter {name}")
        if tuple(state[name].shape) != tuple(p.shape) and [d for d in state[name].shape if d != 1] == [d for d in p.shape if d != 1]:
            state[name] = state[name].reshape(p.shape)                       # the same numbers with or without axes of length 1
        invalidInputError(tuple(state[name].shape) == tuple(p.shape),
                          f"{name}: checkpoint shape {tuple(state[name].shape)} but the configuration gives {tuple(p.shape)}")
    model.load_state_dict(state, strict=True, assign=True)
    model.eval()
    model.requires_grad_(False)
    model.config.dtype = torch_dtype
    if device is not None:
        model = model.to(device)
    return model


# the loaders that go through transformers' Auto classes (load_low_bit builds the architecture from a saved configuration)
def _register():
    from transformers import AutoConfig, AutoModelForCausalLM
    try:
        AutoConfig.register("rumuvik", RumuvikConfig)
        AutoModelForCausalLM.register(RumuvikConfig, RumuvikForCausalLM)
    except ValueError:                                                       # registered already
        pass


_register()
