"""`python bench.py --arch rumuvik`: the Rumuvik design at layer sizes of a real model (random weights), beside a Nikedra -- the
framework's closest model: mixer and feed-forward side by side on two norms, latent attention with one shared rotated key part, grouped
attention, a recurrence with a matrix state -- of equal width, layer runs, heads and feed-forward: prefill and decode throughput
through the public API, and every kernel of the design timed alone against its roofline next to the like kernel of the other designs
at the same sizes.

Timing and rooflines as in bench_mixers.py: CUDA events on the launching stream, 3 warm-up runs, median of 7, a 256 MB buffer
rewritten between runs; algorithmic bytes / the measured copy bandwidth, or algorithmic flops / the measured bf16 GEMM burst
rate (MEASURED_PEAKS.json).  One JSON line on stdout.
"""
import json
import os

from bench_mixers import NEW, PROMPT, ROOT, Timer, throughput
from bench_zubedra import _fill

VOCAB, LAYERS = 32000, 8
ORDER = ("attention", "mlstm", "latent_attention", "mlstm")
LOOP = {"start": 2, "stop": 4, "times": 2}
# per size: width, attention heads / key heads / head size, rotated channels, latent rank / query rank / rotated part, memory heads / key size /
# value size, feed-forward
SIZES = {"2048": dict(width=2048, heads=16, kv_heads=4, dim=128, rot=64, kv_rank=512, q_rank=768, rot_dim=64, m_heads=8, m_dim=128, m_vdim=256, ff=5632),
         "4096": dict(width=4096, heads=32, kv_heads=8, dim=128, rot=64, kv_rank=512, q_rank=1536, rot_dim=64, m_heads=16, m_dim=128, m_vdim=256, ff=11264)}
SCALING = {"factor": 8.0, "original": 2048, "fast": 32.0, "slow": 1.0}


def rumuvik_config(size):
    z = SIZES[size]
    D = z["dim"]
    mixers = {"attention": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": D, "vdim": D, "scale": D ** -0.5, "softcap": 50.0,
                            "rot": {"base": 500000.0, "dims": z["rot"]}},
              "latent_attention": {"heads": z["heads"], "dim": D, "rot_dim": z["rot_dim"], "vdim": D, "kv_rank": z["kv_rank"], "q_rank": z["q_rank"],
                                   "scale": (D + z["rot_dim"]) ** -0.5, "rot": {"base": 10000.0, "dims": z["rot_dim"], "scaling": SCALING}},
              "mlstm": {"heads": z["m_heads"], "dim": z["m_dim"], "vdim": z["m_vdim"], "gate_cap": 15.0}}
    layers = [{"type": ORDER[i % 4], "mixer": mixers[ORDER[i % 4]], "mlp": {"kind": "dense", "ff": z["ff"]}} for i in range(LAYERS)]
    return {"architecture": "Rumuvik", "vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-5}, "embedding": {"scale": 8.0}, "layers": layers, "loop": LOOP}


def nikedra_config(size):
    """as many layers as the other has layer runs; window and chunk hold everything, so that the attention has as much to do; the
    delta rule's heads carry as many state numbers as the matrix memory's"""
    z = SIZES[size]
    D, H = z["dim"], z["heads"]
    latent = {"heads": H, "dim": D, "rot_dim": z["rot_dim"], "vdim": D, "kv_rank": z["kv_rank"], "scale": (D + z["rot_dim"]) ** -0.5, "mask": {"size": 8192},
              "rot": {"base": 10000.0, "dims": z["rot_dim"]}}
    par = {"left": {"heads": H, "kv_heads": z["kv_heads"], "dim": D, "vdim": D, "scale": D ** -0.5, "mask": {"size": 8192},
                    "rot": {"base": 500000.0, "dims": z["rot"], "scaling": SCALING}},
           "right": {"heads": H, "vdim": 64, "state": 128, "groups": 2, "norm_groups": 2, "conv": 4}}
    delta = {"heads": z["m_heads"], "kv_heads": z["m_heads"], "dim": z["m_dim"], "vdim": z["m_vdim"], "conv": 4}
    same = {"attention": ("parallel", par), "latent_attention": ("latent_attention", latent), "mlstm": ("channel_delta", delta)}
    a, b = LOOP["start"], LOOP["stop"]
    runs = list(range(b)) + list(range(a, b)) * (LOOP["times"] - 1) + list(range(b, LAYERS))
    layers = [{"type": same[ORDER[i % 4]][0], "mixer": same[ORDER[i % 4]][1], "mlp": {"kind": "dense", "ff": z["ff"], "limit": 7.0}} for i in runs]
    return {"architecture": "Nikedra", "vocab": VOCAB, "width": z["width"], "canon": {"taps": 4}, "norm": {"eps": 1e-5}, "logit_scale": 1.0, "layers": layers,
            "low_ranks": {str(i): [64, 64] for i, l in enumerate(layers) if l["type"] == "channel_delta"}}


def _expand(model, dev, dtype):
    """the latent expansions get the block form that the loaders give them"""
    import torch
    from ipex_llm_b200.transformers.models.mixers import latent_expansion
    for m in model.modules():
        if hasattr(m, "expand"):
            uk, uv = (torch.randn(m.heads * d, m.kv_rank, dtype=dtype) * m.kv_rank ** -0.5 for d in (m.dim, m.vdim))
            m.expand.weight = torch.nn.Parameter(latent_expansion(uk, uv, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank).to(dev), requires_grad=False)


def build_rumuvik(dev, dtype, size="2048"):
    import torch
    from ipex_llm_b200.transformers.convert import _optimize_pre, _optimize_post
    from ipex_llm_b200.transformers.models.rumuvik import RumuvikConfig, RumuvikForCausalLM
    with torch.device("meta"):
        model = RumuvikForCausalLM(RumuvikConfig(**rumuvik_config(size)))
    _fill(model, dev, dtype, small={"i_bias": -1.0, "f_bias": 4.0})
    _expand(model, dev, dtype)
    return _optimize_post(_optimize_pre(model.eval()))


def build_nikedra(dev, dtype, size="2048"):
    import torch
    from ipex_llm_b200.transformers.convert import _optimize_pre, _optimize_post
    from ipex_llm_b200.transformers.models.nikedra import NikedraConfig, NikedraForCausalLM
    with torch.device("meta"):
        model = NikedraForCausalLM(NikedraConfig(**nikedra_config(size)))
    _fill(model, dev, dtype, small={"A_log": -1.0, "canon": 0.1, "conv_weight": 0.3})
    _expand(model, dev, dtype)
    for layer in model.model.layers:
        layer.dwa.data.fill_(1.0 / layer.dwa.numel())
    return _optimize_post(_optimize_pre(model.eval()))


def kernel_table(dev, dtype, peaks, timer, size):
    """each kernel of the design alone at the layer's sizes (prefill: 1 x PROMPT tokens; decode: 8 rows, one token each, PROMPT
    cached), each followed by the like kernel of the closest designs at the same sizes"""
    import torch
    from ipex_llm_b200.transformers.models import mixer_ops as ops
    z = SIZES[size]
    W, H, G, D, R, Q, Dr, MH, MD, MV, FF, ROT = (z[k] for k in ("width", "heads", "kv_heads", "dim", "kv_rank", "q_rank", "rot_dim", "m_heads", "m_dim", "m_vdim",
                                                               "ff", "rot"))
    hbm, tc = float(peaks["hbm_gbs"]), float(peaks["bf16_tflops"])
    es = torch.empty((), dtype=dtype).element_size()
    rows = []

    def add(name, phase, ms, bytes_=None, flops=None, like_of=None):
        r = {"size": size, "kernel": name, "phase": phase, "us": ms * 1e3}
        if bytes_ is not None:
            r.update(gbs=bytes_ / ms / 1e6, frac_hbm=bytes_ / ms / 1e6 / hbm)
        if flops is not None:
            r.update(tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tc)
        if like_of:
            r["like_of"] = like_of
        rows.append(r)

    rnd = lambda *s: torch.randn(*s, device=dev).to(dtype)                                  # noqa: E731
    vec = lambda *s: (torch.rand(*s, device=dev) + 0.5).to(dtype)                            # noqa: E731
    freqs = lambda n, base: torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=torch.float64, device=dev)      # noqa: E731
    for phase, B, S, held in (("prefill", 1, PROMPT, 0), ("decode", 8, 1, PROMPT)):
        N, L = B * S, held + S
        pad = torch.zeros(B, dtype=torch.int32, device=dev)
        # the stream
        x, yf, ya, yb, x0 = torch.randn(N, W, device=dev), torch.randn(N, W, device=dev), rnd(N, W), rnd(N, W), torch.randn(N, W, device=dev)
        wa, wb, one = vec(W), vec(W), vec(1)
        add("sum_residual_norms (32-bit sum, two zero-centred vector norms)", phase,
            timer(lambda: ops.sum_residual_norms(x, [yf], dtype, 1e-5, gain1=wa, gain2=wb, gain_add=1.0)), N * W * (12 + 2 * es))
        add("sum_residual_norms (the same and the embedding output)", phase,
            timer(lambda: ops.sum_residual_norms(x, [yf, x0], dtype, 1e-5, gain1=wa, gain2=wb, gain_add=1.0)), N * W * (16 + 2 * es))
        add("sum_residual_norms (two 16-bit sums, two scalar norms)", phase,
            timer(lambda: ops.sum_residual_norms(x, [ya, yb], dtype, 1e-5, gain1=one, gain2=one)), N * W * (8 + 4 * es), like_of="sum_residual_norms")
        # attention with rotated values
        P = (H + 2 * G) * D
        proj, ks, vs = rnd(B, S, P), rnd(B, G, L, D), rnd(B, G, L, D)
        fk, fv = freqs(ROT, 500000.0), freqs(D, 500000.0)
        add("rotary_table", phase, timer(lambda: ops.rotary_table(fv, 1.0, B, S, held, 0, pad)), N * D * 4)
        tk, tv = ops.rotary_table(fk, 1.0, B, S, held, 0, pad), ops.rotary_table(fv, 1.0, B, S, held, 0, pad)
        st = (G * L * D, D, L * D)
        add("rope_qk_prepare (tables, rotated values)", phase,
            timer(lambda: ops.rope_qk_prepare(proj, 0, H * D, (H + G) * D, H, G, D, D, D, 0, 0, ROT, None, 1.0, ks, st, vs, st, held, 0, pad, table=tk, v_table=tv)),
            N * (2 * P * es + ROT * 4 + D * 4))
        add("rope_qk_prepare (angles formed per head)", phase,
            timer(lambda: ops.rope_qk_prepare(proj, 0, H * D, (H + G) * D, H, G, D, D, D, 0, 0, ROT, fk, 1.0, ks, st, vs, st, held, 0, pad)),
            N * 2 * P * es, like_of="rope_qk_prepare (tables, rotated values)")
        q, zero, out = rnd(N, H * D), torch.zeros(H, dtype=dtype, device=dev), torch.empty(N, H * D + FF, dtype=dtype, device=dev)
        kview, vview = ks.permute(0, 2, 1, 3), vs.permute(0, 2, 1, 3)
        work = dict(flops=4.0 * D * (S * (S + 1) / 2) * H * B) if S > 1 else dict(bytes_=B * G * L * 2 * D * es)
        add("softmax_attention (capped, a one in the denominator, turned back)", phase,
            timer(lambda: ops.softmax_attention(q, kview, vview, B, S, H, held, 0, pad, 0, D ** -0.5, out=out, softcap=50.0, sink=zero, back=tv)), **work)
        add("softmax_attention (capped, a sink)", phase,
            timer(lambda: ops.softmax_attention(q, kview, vview, B, S, H, held, 0, pad, 0, D ** -0.5, out=out, softcap=50.0, sink=zero)),
            like_of="softmax_attention (capped, a one in the denominator, turned back)", **work)
        add("softmax_attention (plain)", phase, timer(lambda: ops.softmax_attention(q, kview, vview, B, S, H, held, 0, pad, 0, D ** -0.5, out=out)),
            like_of="softmax_attention (capped, a one in the denominator, turned back)", **work)
        # latent attention
        lp, store, wq, wc = rnd(B, S, Q + R + Dr), rnd(B, L, R + Dr), vec(Q), vec(R)
        add("rms_norm_columns (query latent)", phase, timer(lambda: ops.rms_norm_columns(lp, 0, Q, wq, 1e-5, held, 0, pad)), N * Q * 2 * es)
        lstore = rnd(B, L, R)
        add("latent_prepare (query and key latent)", phase, timer(lambda: ops.latent_prepare(lp, 0, Q, wq, Q, R, wc, 1e-5, lstore, held, 0, pad)),
            N * (Q + R) * 2 * es, like_of="rms_norm_columns")
        lq, fl = rnd(B, S, H * (D + Dr)), freqs(Dr, 10000.0)
        tl = ops.rotary_table(fl, 1.2, B, S, held, 0, pad)
        ls = (L * (R + Dr), R + Dr, 0)
        move = N * (2 * (H * (D + Dr) + R + Dr) * es)
        add("rope_qk_prepare (latent rows, neighbouring pairs, tables)", phase,
            timer(lambda: ops.rope_qk_prepare(lq, 0, Q, 0, H, 1, D + Dr, R + Dr, 0, D, R, Dr, None, 1.0, store, ls, None, None, held, 0, pad, eps=1e-5, k_norm_w=wc,
                                              k_norm_cols=R, table=tl, interleaved=True, kv_proj=lp)), move + N * Dr * 4)
        both = rnd(B, S, H * (D + Dr) + R + Dr)
        add("rope_qk_prepare (latent rows, angles formed per head)", phase,
            timer(lambda: ops.rope_qk_prepare(both, 0, H * (D + Dr), 0, H, 1, D + Dr, R + Dr, 0, D, R, Dr, fl, 1.2, store, ls, None, None, held, 0, pad, eps=1e-5,
                                              k_norm_w=wc, k_norm_cols=R)), move, like_of="rope_qk_prepare (latent rows, neighbouring pairs, tables)")
        if S > 1:
            kvx = rnd(B, L, H * (2 * D + Dr))
            k4, v4 = kvx[..., :H * (D + Dr)].view(B, L, H, D + Dr), kvx[..., H * (D + Dr):].view(B, L, H, D)
            lq2 = lq.view(N, -1)
            add("softmax_attention (expanded latents)", phase, timer(lambda: ops.softmax_attention(lq2, k4, v4, B, S, H, held, 0, pad, 0, 0.07, out=out)),
                flops=2.0 * (2 * D + Dr) * (S * (S + 1) / 2) * H * B)
            add("softmax_attention (expanded latents under a window of 8192)", phase,
                timer(lambda: ops.softmax_attention(lq2, k4, v4, B, S, H, held, 0, pad, 8192, 0.07, out=out)), flops=2.0 * (2 * D + Dr) * (S * (S + 1) / 2) * H * B,
                like_of="softmax_attention (expanded latents)")
        else:
            qa, rows_ = rnd(N, H * (R + Dr)), store.unsqueeze(2)
            add("softmax_attention (on the latent cache)", phase,
                timer(lambda: ops.softmax_attention(qa, rows_, rows_[..., :R], B, S, H, held, 0, pad, 0, 0.07)), B * L * (R + Dr) * es)
            add("softmax_attention (on the latent cache, window of 8192)", phase,
                timer(lambda: ops.softmax_attention(qa, rows_, rows_[..., :R], B, S, H, held, 0, pad, 8192, 0.07)), B * L * (R + Dr) * es,
                like_of="softmax_attention (on the latent cache)")
        # matrix memory
        MP = MH * (2 * MD + 2 * MV) + 2 * MH
        mp, state, norm, top = rnd(B, S, MP), *(torch.zeros(*s, device=dev) for s in ((B, MH, MD, MV), (B, MH, MD), (B, MH, MV + 1)))
        bi, bf = rnd(MH) - 1.0, rnd(MH) + 4.0
        off_i = MP - 2 * MH
        rec = N * (MH * (2 * MD + MV) * es + MH * MV * 4) + 2 * B * MH * MD * MV * 4
        add("mlstm", phase, timer(lambda: ops.mlstm(mp, 0, MH * MD, 2 * MH * MD, off_i, off_i + MH, MH, MD, MV, bi, bf, 15.0, 1e-6, state, norm, top, held, None)),
            rec + N * MH * (2 * es + 4), flops=4.0 * N * MH * MD * (MV + 1))
        decay, zz = torch.full((MH,), 0.99, device=dev), rnd(B, S, MH * MD)
        add("constant_decay_attention", phase, timer(lambda: ops.constant_decay_attention(mp, 0, MH, MD, MV, decay, state, held, None)), rec,
            flops=4.0 * N * MH * MD * MV, like_of="mlstm")
        add("gated_linear_attention", phase, timer(lambda: ops.gated_linear_attention(mp, MH, MD, MV, zz, 16.0, state, held, None)), rec + N * MH * MD * es,
            flops=4.0 * N * MH * MD * MV, like_of="mlstm")
        o, below, gw, mp2 = torch.randn(N, MH, MV, device=dev), torch.rand(N, MH, device=dev) + 0.5, vec(MH * MV), mp.view(N, MP)
        off_g = MH * (2 * MD + MV)
        add("gated_rms_norm (over the denominators)", phase,
            timer(lambda: ops.gated_rms_norm(o, mp2, off_g, gw, 1e-5, out, 0, 1.0, sigmoid=True, below=below)), N * MH * MV * (4 + 2 * es) + N * MH * 4)
        add("gated_rms_norm", phase, timer(lambda: ops.gated_rms_norm(o, mp2, off_g, gw, 1e-5, out, 0, 1.0, sigmoid=True)), N * MH * MV * (4 + 2 * es),
            like_of="gated_rms_norm (over the denominators)")
        # feed-forward
        gu = rnd(N, 2 * FF)
        add("gelu_tanh_mul (into a column range)", phase, timer(lambda: ops.gelu_tanh_mul(gu, FF, out=out[:, H * D:])), N * FF * 3 * es)
        add("clamped_glu", phase, timer(lambda: ops.clamped_glu(gu, FF, 7.0)), N * FF * 3 * es, like_of="gelu_tanh_mul")
    return rows


def run(args):
    import torch
    dev = torch.device("cuda", 0)
    torch.cuda.set_device(dev)
    dtype = torch.bfloat16
    try:
        peaks = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
        src = "MEASURED_PEAKS.json"
    except (OSError, ValueError):
        peaks, src = {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}, "fallback"
    timer = Timer(dev)
    out = {"arch": "rumuvik", "dtype": "bf16", "data": "synthetic (random weights)",
           "peaks": {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "source": src},
           "config": {"sizes": SIZES, "layers": LAYERS, "layer_order": ORDER, "loop": LOOP, "vocab": VOCAB, "prompt": PROMPT, "new_tokens": NEW,
                      "cache": "256 MB rewritten between timed runs"}, "kernels": []}
    for size in [s for s in SIZES if not getattr(args, "sizes", None) or s in args.sizes.split(",")]:
        models = [("rumuvik_", build_rumuvik)] + ([] if args.no_compare else [("nikedra_equal_size_", build_nikedra)])
        for name, build in models:
            model = build(dev, dtype, size)
            out[name + size] = [throughput(model, dev, timer, b) for b in (1, 8)]
            out[name + size + "_recorded_step_failed"] = model.__dict__.get("_b200_state_graph_failed")
            model.__dict__.pop("_b200_state_graphs", None)
            del model
            torch.cuda.empty_cache()
        out["kernels"] += kernel_table(dev, dtype, peaks, timer, size)
    out["nikedra_equal_size_note"] = "bf16, same width / layer runs / heads / latent ranks / state sizes / feed-forward width; window and chunk hold everything"
    print(json.dumps(out))
