"""Bugipel: a decoder-only design of pre-norm layers (RMS norms with a weight vector), a stretch of which runs several times in a
row with the same weights.  In front of every pass over that stretch the stream is projected anew from [stream ; embedding output]
and a vector that belongs to the pass is added; every pass keeps a cache or state of its own.  A layer's mixer is one of

* ``lightning``: linear attention with one constant decay per head, silu on q, k and v, an RMS norm over all heads' read-outs
  together and a sigmoid gate per channel;
* ``parallel``: two mixers on the same input, added with a constant each.  ``left`` is grouped softmax attention whose values are its
  keys as projected; queries and keys are rotated, then divided by their root mean square per head (no weight); the softmax's
  denominator also holds a one (a sink of score 0 that has no value); a sigmoid gate per channel.  ``right`` is the delta rule with
  a decay per key channel of ``models/mixers.py``;

and its feed-forward (optional) is ``down(gelu(up h))`` with the exact gelu.  The output head is the embedding table.

No library ships this model.  The module tree, the configuration reader and the checkpoint's name map live here; the state in
``transformers/kv.py`` (``DynamicStateCache``: one key/value store, matrix state and convolution tail per layer RUN), the kernels in
``csrc/mixers`` behind ``ggml/model/mixers_cpp.py``.  The projections are ``nn.Linear`` modules, so the low-bit conversion treats
them like any other model's.  The residual stream, every norm, rotary angles, attention scores and weights and everything inside
the recurrences are 32-bit whatever the model's dtype.
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
from ipex_llm_b200.transformers.models.mixers import ChannelDeltaMixer, Constants, Rotary, Weight, channel_delta, linear_f32, plain_linears
from ipex_llm_b200.transformers.models.utils import read_safetensors
from ipex_llm_b200.utils.common import invalidInputError

OVERLAP_MIN_TOKENS = 256      # from this many new tokens on, a parallel layer's two branches run on two streams


class BugipelConfig(PreTrainedConfig):
    """config.json of the design: ``vocab``, ``width``, ``layers`` (per layer: ``type``, ``mixer`` sizes and constants, ``mlp`` or
    null), ``loop`` (``start``, ``stop``, ``times``; optional), ``norm.eps``.  ``low_ranks`` (per parallel layer: the ranks of the
    delta rule's decay and gate projections) is not a key of the design's config.json: the loader reads it off the checkpoint's
    shapes, and it is kept so that a saved model can be rebuilt from its configuration alone."""
    model_type = "bugipel"

    def __init__(self, vocab=256, width=64, layers=None, loop=None, norm=None, architecture="Bugipel", low_ranks=None, **kwargs):
        self.vocab, self.width = int(vocab), int(width)
        self.layers = layers or []
        self.loop = loop
        self.norm = norm or {"eps": 1e-5}
        self.architecture = architecture
        self.low_ranks = {str(k): [int(v[0]), int(v[1])] for k, v in (low_ranks or {}).items()}
        # the head shares the embedding's parameter at load time; a converted head is a low-bit copy, which tying by the library
        # would overwrite
        kwargs["tie_word_embeddings"] = False
        super().__init__(**kwargs)
        self.vocab_size, self.hidden_size, self.num_hidden_layers = self.vocab, self.width, len(self.layers)
        self.use_cache = True

    @property
    def norm_eps(self):
        return float(self.norm["eps"])

    @property
    def passes(self):
        return int(self.loop.get("times", 0)) if self.loop else 0

    def layer_runs(self):
        """[(layer, t)]: the layers in the order in which they run; t is the number of the pass that starts with this run, else None"""
        n = len(self.layers)
        if not self.passes:
            return [(i, None) for i in range(n)]
        start, stop = int(self.loop["start"]), int(self.loop["stop"])
        invalidInputError(0 <= start < stop <= n, "loop: start .. stop - 1 must name layers")
        looped = [(i, t if i == start else None) for t in range(self.passes) for i in range(start, stop)]
        return [(i, None) for i in range(start)] + looped + [(i, None) for i in range(stop, n)]


class LightningMixer(nn.Module):
    """``q_proj`` / ``k_proj`` / ``v_proj`` / ``g_proj`` become one ``in_proj`` when ``merge_projections`` has run"""

    def __init__(self, width, m):
        super().__init__()
        self.heads, self.dim, self.vdim = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        invalidInputError(len(m["decay"]) == self.heads, "a lightning mixer has one decay per head")
        self.decay = Constants(m["decay"])
        qk, v = self.heads * self.dim, self.heads * self.vdim
        self.q_proj, self.k_proj = nn.Linear(width, qk, bias=False), nn.Linear(width, qk, bias=False)
        self.v_proj, self.g_proj = nn.Linear(width, v, bias=False), nn.Linear(width, v, bias=False)
        self.norm = Weight(v)
        self.o_proj = nn.Linear(v, width, bias=False)


class KeyValueAttention(nn.Module):
    """grouped attention whose values are its keys as projected (before rotation and norm)"""

    def __init__(self, width, m):
        super().__init__()
        self.heads, self.kv_heads, self.dim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
        invalidInputError(self.kv_heads >= 1 and self.heads % self.kv_heads == 0, "heads must be a multiple of kv_heads")
        invalidInputError(int(m.get("vdim", self.dim)) == self.dim, "the values are the keys: vdim must equal dim")
        self.scale = float(m["scale"])
        self.rotary = Rotary(m["rot"])
        invalidInputError(self.rotary.dims <= self.dim, "rotary dims exceed the head size")
        self.sink = Constants([0.0] * self.heads)             # the score of the one in the softmax's denominator
        self.q_proj = nn.Linear(width, self.heads * self.dim, bias=False)
        self.k_proj = nn.Linear(width, self.kv_heads * self.dim, bias=False)
        self.g_proj = nn.Linear(width, self.heads * self.dim, bias=False)
        self.o_proj = nn.Linear(self.heads * self.dim, width, bias=False)


class ParallelMixer(nn.Module):
    """``in_proj`` (both branches' projections of the input) and ``out_proj`` (both output projections over the concatenated branch
    outputs: their sum happens in the accumulator of one product) appear when ``merge_projections`` has run"""

    def __init__(self, width, m, ranks):
        super().__init__()
        self.left, self.right = KeyValueAttention(width, m["left"]), ChannelDeltaMixer(width, m["right"], ranks)
        self.left_scale, self.right_scale = float(m["left_scale"]), float(m["right_scale"])


class GeluMLP(nn.Module):
    """down(gelu(up h)) with the exact gelu, no biases"""

    def __init__(self, width, m):
        super().__init__()
        invalidInputError(m.get("kind", "dense") == "dense", f"unknown feed-forward kind {m.get('kind')}")
        self.up_proj, self.down_proj = nn.Linear(width, int(m["ff"]), bias=False), nn.Linear(int(m["ff"]), width, bias=False)

    def forward(self, h):
        return self.down_proj(ops.gelu_erf(self.up_proj(h)))


class BugipelLayer(nn.Module):
    def __init__(self, config: BugipelConfig, index):
        super().__init__()
        lc, w = config.layers[index], config.width
        self.kind = lc["type"]
        invalidInputError(self.kind in ("lightning", "parallel"), f"unknown layer type {self.kind}")
        self.norm1 = Weight(w)
        if self.kind == "lightning":
            self.mixer = LightningMixer(w, lc["mixer"])
        else:
            self.mixer = ParallelMixer(w, lc["mixer"], config.low_ranks.get(str(index), [1, 1]))
        self.mlp = None
        if lc.get("mlp") is not None:
            self.norm2 = Weight(w)
            self.mlp = GeluMLP(w, lc["mlp"])


def merge_projections(module: nn.Module, row_multiple: int = 0):
    """every projection that reads a mixer's input becomes one ``in_proj``, a parallel mixer's two output projections one
    ``out_proj``; ``row_multiple``: see ``zero_rows`` (the kernels address columns by offset, the extra ones are never read)"""
    if isinstance(module, ParallelMixer) and not hasattr(module, "in_proj"):
        l, r = module.left, module.right
        parts = [l.q_proj, l.k_proj, l.g_proj] + [getattr(r, n) for n in r.PARTS]
        module.in_proj = merge_linear(parts + zero_rows(l.q_proj, sum(p.weight.shape[0] for p in parts), row_multiple))
        module.out_proj = merge_linear_inputs([l.o_proj, r.o_proj])
        del l.q_proj, l.k_proj, l.g_proj, l.o_proj, r.o_proj
        for n in r.PARTS:
            delattr(r, n)
    elif isinstance(module, LightningMixer) and not hasattr(module, "in_proj"):
        parts = [module.q_proj, module.k_proj, module.v_proj, module.g_proj]
        module.in_proj = merge_linear(parts + zero_rows(module.q_proj, sum(p.weight.shape[0] for p in parts), row_multiple))
        del module.q_proj, module.k_proj, module.v_proj, module.g_proj


class BugipelModel(nn.Module):
    def __init__(self, config: BugipelConfig):
        super().__init__()
        self.config = config
        w = config.width
        self.embed_tokens = nn.Embedding(config.vocab, w)
        if config.passes:
            self.loop_in = nn.Linear(2 * w, w, bias=False)
            self.loop_step = nn.Parameter(torch.zeros(config.passes, w))
        self.layers = nn.ModuleList([BugipelLayer(config, i) for i in range(len(config.layers))])
        self.norm = Weight(w)


class BugipelForCausalLM(PreTrainedModel, GenerationMixin):
    config_class = BugipelConfig
    base_model_prefix = "model"
    _no_split_modules = ["BugipelLayer"]
    _supports_attention_backend = False
    main_input_name = "input_ids"

    def __init__(self, config: BugipelConfig):
        super().__init__(config)
        self.model = BugipelModel(config)
        self.lm_head = nn.Linear(config.width, config.vocab, bias=False)
        self.collect_residual = None          # a list: gets the residual stream after every layer run (debugging aid)
        self.attention_tensor_cores = True    # 16-bit models: prompts take the tensor-core attention kernel
        self.overlap_branches = True          # prompts: a parallel layer's branches read the same input, so they run side by side
        self._side_stream = None

    def _init_weights(self, module):
        pass

    def get_input_embeddings(self):
        return self.model.embed_tokens

    def get_output_embeddings(self):
        return self.lm_head

    def share_head(self):
        """the output head is the embedding table: one parameter for both"""
        self.lm_head.weight = self.model.embed_tokens.weight
        return self

    # ---- mixers (h: the normalised input in the model's dtype, [N, W]); each returns [N, W]
    def _lightning(self, mx, h, st, B, S, cache):
        invalidInputError(hasattr(mx, "in_proj"), "the mixers' projections are merged at load time (merge_projections)")
        H, D, Dv, N = mx.heads, mx.dim, mx.vdim, B * S
        proj = mx.in_proj(h)                                                 # q | k | v | gate
        state = st.rec.matrix(B, H, D, Dv, h.device)
        o = ops.constant_decay_attention(proj.view(B, S, -1), 0, H, D, Dv, mx.decay.on(h.device), state, cache.seen,
                                         cache.pad if cache.seen == 0 else None)
        out = torch.empty(N, H * Dv, dtype=h.dtype, device=h.device)
        ops.gated_rms_norm(o.view(N, 1, H * Dv), proj, H * (2 * D + Dv), mx.norm.weight, self.config.norm_eps, out, 0, 1.0, sigmoid=True)
        return mx.o_proj(out)

    def _left(self, mx, proj, out, st, B, S, cache):
        """attention into the first columns of ``out``"""
        l = mx.left
        H, G, D = l.heads, l.kv_heads, l.dim
        off_k = H * D
        off_g = off_k + G * D
        kv = st.kv
        like = torch.empty((B, G, 0, D), dtype=proj.dtype, device=proj.device)
        k_store, v_store, held = kv.slots(like, like, S)
        shift = cache.seen - held                                            # storage index + shift = slot number
        # a recorded decode step reads the length from the device (the value given here is the one at recording time)
        dyn = kv.length_dev if (cache.frozen and S == 1) else None
        cap = kv.capacity()
        strides = (G * cap * D, D, cap * D)
        q = ops.rope_qk_prepare(proj.view(B, S, -1), 0, off_k, off_k, H, G, D, D, D, 0, 0, l.rotary.dims, l.rotary.inv_freq(proj.device), l.rotary.amp,
                                k_store, strides, v_store, strides, held, shift, cache.pad, eps=self.config.norm_eps, dyn=dyn, unit_rms=True)
        kv.commit(S)
        ops.softmax_attention(q, k_store.permute(0, 2, 1, 3), v_store.permute(0, 2, 1, 3), B, S, H, held, shift, cache.pad, 0, l.scale, out=out,
                              dyn=dyn, tensor_cores=self.attention_tensor_cores, sink=l.sink.on(proj.device, proj.dtype))
        ops.sigmoid_gate(out[:, :H * D], proj, off_g, 1, scale=mx.left_scale)

    def _parallel(self, mx, h, st, B, S, cache):
        invalidInputError(hasattr(mx, "in_proj"), "the mixers' projections are merged at load time (merge_projections)")
        l, r = mx.left, mx.right
        proj = mx.in_proj(h)                                                 # left q | k | gate | right q | k | v | beta | ranks
        left_cols = l.heads * l.dim
        off_r = 2 * left_cols + l.kv_heads * l.dim
        out = torch.empty(B * S, left_cols + r.heads * r.vdim, dtype=h.dtype, device=h.device)
        eps, dev = self.config.norm_eps, h.device
        if (self.overlap_branches and S > 1 and B * S >= OVERLAP_MIN_TOKENS and dev.type == "cuda" and not torch.cuda.is_current_stream_capturing()
                and plain_linears(self)):
            # the recurrence walks its tokens on a fraction of the SMs, the attention takes the rest.  What outlives the call
            # (state, convolution tail) is allocated on the main stream
            st.rec.matrix(B, r.heads, r.dim, r.vdim, dev)
            st.rec.tails(B, r.taps, r.conv_channels, h.dtype, dev, key="mixer")
            main = torch.cuda.current_stream(dev)
            if self._side_stream is None or self._side_stream.device != dev:
                self._side_stream = torch.cuda.Stream(dev)
            side = self._side_stream
            side.wait_stream(main)
            with torch.cuda.stream(side):
                channel_delta(r, proj, off_r, st.rec, B, S, cache, eps, out, left_cols, mx.right_scale)
            self._left(mx, proj, out, st, B, S, cache)
            main.wait_stream(side)
        else:
            self._left(mx, proj, out, st, B, S, cache)
            channel_delta(r, proj, off_r, st.rec, B, S, cache, eps, out, left_cols, mx.right_scale)
        return mx.out_proj(out)

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
        W = cfg.width
        dev, dtype = core.embed_tokens.weight.device, core.embed_tokens.weight.dtype
        eps = cfg.norm_eps
        cache = past_key_values
        if not isinstance(cache, DynamicStateCache):
            invalidInputError(cache is None or cache.get_seq_length() == 0, "a filled cache of another class cannot be continued")
            cache = DynamicStateCache()
        if cache.seen == 0:                                                  # a batch's first call: the mask gives the padding
            cache.start(attention_mask, B, S, dev)
        invalidInputError(cache.pad.shape[0] == B, "batch size differs from the cache's")
        input_ids = input_ids.to(dev).contiguous()
        runs = cfg.layer_runs()
        # padding only occurs in a batch's first call; later calls (a replayed step among them, whose slot number is the one at
        # recording time) say so by passing no padding
        x, x0 = ops.embed_pair(core.embed_tokens.weight, 1.0, None, 0, 0, 0, input_ids, None, cache.seen, cache.pad if cache.seen == 0 else None, dtype)
        joint = None
        if cfg.passes:                                                       # [stream ; embedding output]: what a pass's projection reads
            joint = torch.empty(B * S, 2 * W, dtype=dtype, device=dev)
            joint.view(B * S, 2, W).copy_(x0.unsqueeze(1))

        # the last norm rides along with the last residual update when every position's logits are wanted
        keep_all = S == 1 or (isinstance(logits_to_keep, int) and logits_to_keep == 0)

        def hand_on(ys, run):
            """x += ys in front of layer run number ``run``; returns the normalised stream that this run's mixer reads"""
            if run == len(runs):
                return ops.sum_residual_norms(x, ys, dtype, eps, gain1=core.norm.weight if keep_all else None)[0]
            li, t = runs[run]
            gain = core.layers[li].norm1.weight
            if t is None:
                return ops.sum_residual_norms(x, ys, dtype, eps, gain1=gain)[0]
            if ys:
                ops.sum_residual_norms(x, ys, dtype, eps, x_copy=joint[:, :W])
            return ops.sum_residual_norms(x, [linear_f32(core.loop_in, joint)], dtype, eps, replace=True, vec=core.loop_step[t], gain1=gain)[0]

        h = hand_on([], 0)
        for run, (li, _) in enumerate(runs):
            layer = core.layers[li]
            if layer.kind == "lightning":
                y = self._lightning(layer.mixer, h, cache.run_state(run), B, S, cache)
            else:
                y = self._parallel(layer.mixer, h, cache.run_state(run, window=0), B, S, cache)
            if layer.mlp is not None:
                h = ops.sum_residual_norms(x, [y], dtype, eps, gain1=layer.norm2.weight)[0]
                y = layer.mlp(h)
            if self.collect_residual is not None:
                self.collect_residual.append((x + y).view(B, S, -1))
            h = hand_on([y], run + 1)
        cache.advance(S)
        if keep_all:
            hn = h.view(B, S, W)
        else:
            idx = slice(-logits_to_keep, None) if isinstance(logits_to_keep, int) else logits_to_keep.to(dev)
            hn = ops.rms_norm_rows(x.view(B, S, W)[:, idx, :].contiguous(), None, core.norm.weight, eps, dtype)
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
def checkpoint_key_map(config: BugipelConfig):
    """the model's parameter names -> the checkpoint's tensor names: one name, or a list of them (concatenated by rows)"""
    m = {"model.embed_tokens.weight": "embed", "lm_head.weight": "embed", "model.norm.weight": "final.norm"}
    if config.passes:
        m["model.loop_in.weight"], m["model.loop_step"] = "loop.in", "loop.step"
    for i, lc in enumerate(config.layers):
        d, s = f"model.layers.{i}.", f"l{i}."
        m[d + "norm1.weight"] = s + "norm1"
        dm, sm = d + "mixer.", s + "mix."
        if lc["type"] == "lightning":
            for n in ("q", "k", "v", "g", "o"):
                m[dm + n + "_proj.weight"] = sm + n
            m[dm + "norm.weight"] = sm + "norm"
        else:
            for n in ("q", "k", "g", "o"):
                m[dm + "left." + n + "_proj.weight"] = sm + "left." + n
            dr, sr = dm + "right.", sm + "right."
            for n in ("q", "k", "v", "b", "a1", "a2", "g1", "g2", "o"):
                m[dr + n + "_proj.weight"] = sr + n
            m[dr + "conv_weight"] = [sr + "q.conv", sr + "k.conv", sr + "v.conv"]
            m[dr + "A_log"], m[dr + "dt_bias"], m[dr + "norm.weight"] = sr + "A_log", sr + "dt_bias", sr + "norm"
        if lc.get("mlp") is not None:
            m[d + "norm2.weight"] = s + "norm2"
            m[d + "mlp.up_proj.weight"], m[d + "mlp.down_proj.weight"] = s + "mlp.up", s + "mlp.down"
    return m


def load_pretrained(model_dir, torch_dtype=None, device=None):
    """config.json + model.safetensors of the design -> a ``BugipelForCausalLM``.  Sizes that config.json does not state (the ranks
    of the delta rule's decay and gate projections) come from the tensors' shapes."""
    with open(os.path.join(model_dir, "config.json")) as f:
        raw = json.load(f)
    tensors = read_safetensors(os.path.join(model_dir, "model.safetensors"))
    if "low_ranks" not in raw:
        raw["low_ranks"] = {str(i): [tensors[f"l{i}.mix.right.{n}"].shape[0] for n in ("a1", "g1")]
                            for i, lc in enumerate(raw.get("layers", []))
                            if lc["type"] == "parallel" and all(f"l{i}.mix.right.{n}" in tensors for n in ("a1", "g1"))}
    config = BugipelConfig(**raw)
    if torch_dtype in (None, "auto"):
        torch_dtype = tensors["embed"].dtype
    with torch.device("meta"):
        model = BugipelForCausalLM(config)
    state = {}
    for dst, src in checkpoint_key_map(config).items():
        names = [src] if isinstance(src, str) else list(src)
        missing = [s for s in names if s not in tensors]
        invalidInputError(not missing, f"the checkpoint has no tensor {missing}")
        t = tensors[src] if isinstance(src, str) else torch.cat([tensors[s] for s in src], dim=0)
        state[dst] = t.to(torch_dtype)
    for name, p in model.named_parameters():
        invalidInputError(name in state, f"no checkpoint tensor for parameter {name}")
        if tuple(state[name].shape) != tuple(p.shape) and [d for d in state[name].shape if d != 1] == [d for d in p.shape if d != 1]:
            state[name] = state[name].reshape(p.shape)                       # the same numbers with or without axes of length 1
        invalidInputError(tuple(state[name].shape) == tuple(p.shape),
                          f"{name}: checkpoint shape {tuple(state[name].shape)} but the configuration gives {tuple(p.shape)}")
    model.load_state_dict(state, strict=True, assign=True)
    model.share_head()
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
        AutoConfig.register("bugipel", BugipelConfig)
        AutoModelForCausalLM.register(BugipelConfig, BugipelForCausalLM)
    except ValueError:                                                       # registered already
        pass


_register()
