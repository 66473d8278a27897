"""`python bench.py --arch bugipel`: the Bugipel design at layer sizes of a real model (random weights), beside a Zafepel -- the
framework's closest model: layers of attention beside a delta rule and layers of linear attention, a stretch of them run twice -- of
equal width, depth, layer runs, heads and feed-forward: prefill and decode throughput through the public API, and every kernel of
the design timed alone against its roofline next to the like kernel of the Zafepel path at the same sizes.

Timing and rooflines as in bench_mixers.py: CUDA events on the launching stream, 3 warm-up runs, median of 7, a 256 MB buffer
rewritten between runs; algorithmic bytes / the measured copy bandwidth, or algorithmic flops / the measured bf16 GEMM burst
rate (MEASURED_PEAKS.json).  One JSON line on stdout.
"""
import json
import os

from bench_mixers import NEW, PROMPT, ROOT, Timer, throughput
from bench_zubedra import _fill

VOCAB, LAYERS, CONV = 32000, 8, 4
LOOP = {"start": 2, "stop": 4, "times": 2}
# per size: width, attention heads / key heads / head size, rotated channels, delta rule heads / key heads, its low ranks, linear attention
# heads / key size / value size, feed-forward
SIZES = {"2048": dict(width=2048, heads=16, kv_heads=4, dim=128, rot=64, d_heads=16, d_kv=4, rank=64, l_heads=8, l_dim=128, l_vdim=256, ff=5632),
         "4096": dict(width=4096, heads=32, kv_heads=8, dim=128, rot=64, d_heads=32, d_kv=8, rank=128, l_heads=16, l_dim=128, l_vdim=256, ff=11264)}


def _delta(z):
    return {"heads": z["d_heads"], "kv_heads": z["d_kv"], "dim": z["dim"], "vdim": z["dim"], "conv": CONV}


def bugipel_config(size):
    z = SIZES[size]
    light = {"heads": z["l_heads"], "dim": z["l_dim"], "vdim": z["l_vdim"], "decay": [1.0 - 2.0 ** -(5 + 8 * h / z["l_heads"]) for h in range(z["l_heads"])]}
    par = {"left": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                    "rot": {"base": 500000.0, "dims": z["rot"]}}, "left_scale": 0.7, "right": _delta(z), "right_scale": 0.7}
    layers = [{"type": "parallel" if i % 2 == 0 else "lightning", "mixer": par if i % 2 == 0 else light, "mlp": {"kind": "dense", "ff": z["ff"]}}
              for i in range(LAYERS)]
    return {"architecture": "Bugipel", "vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-5}, "layers": layers, "loop": LOOP,
            "low_ranks": {str(i): [z["rank"], z["rank"]] for i in range(0, LAYERS, 2)}}


def zafepel_config(size):
    """the window holds everything, so that the attention has as much to do"""
    z = SIZES[size]
    par = {"left": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5, "mask": {"size": 8192},
                    "rot": {"base": 10000.0, "dims": z["rot"]}}, "left_scale": 1.0, "right": _delta(z), "right_scale": 1.0}
    gla = {"heads": z["l_heads"], "dim": z["l_dim"], "vdim": z["l_vdim"], "tau": 16.0}
    layers = [{"type": "parallel" if i % 2 == 0 else "gla", "mixer": par if i % 2 == 0 else gla, "mlp": {"kind": "dense", "ff": z["ff"]}} for i in range(LAYERS)]
    return {"architecture": "Zafepel", "vocab": VOCAB, "width": z["width"], "norm": {"eps": 1e-5}, "layers": layers, "loop": LOOP, "logit_softcap": 30.0}


def build_bugipel(dev, dtype, size="2048"):
    import torch
    from ipex_llm_b200.transformers.convert import _optimize_pre, _optimize_post
    from ipex_llm_b200.transformers.models.bugipel import BugipelConfig, BugipelForCausalLM
    with torch.device("meta"):
        model = BugipelForCausalLM(BugipelConfig(**bugipel_config(size)))
    _fill(model, dev, dtype, small={"A_log": -1.0, "conv_weight": 0.3, "loop_step": 0.1})
    return _optimize_post(_optimize_pre(model.share_head().eval()))


def build_zafepel(dev, dtype, size="2048"):
    import torch
    from ipex_llm_b200.transformers.convert import _optimize_pre, _optimize_post
    from ipex_llm_b200.transformers.models.zafepel import ZafepelConfig, ZafepelForCausalLM
    with torch.device("meta"):
        model = ZafepelForCausalLM(ZafepelConfig(**zafepel_config(size)), {i: 16 for i in range(1, LAYERS, 2)})
    _fill(model, dev, dtype, ones=("weight", "alpha"), small={"A_log": -1.0, "conv_weight": 0.3, "loop_step": 0.1})
    return _optimize_post(_optimize_pre(model.eval()))


def kernel_table(dev, dtype, peaks, timer, size):
    """each kernel of the design alone at the layer's sizes (prefill: 1 x PROMPT tokens; decode: 8 rows, one token each, PROMPT
    cached), each followed by the like kernel of the Zafepel path at the same sizes"""
    import torch
    from ipex_llm_b200.transformers.models import mixer_ops as ops
    from ipex_llm_b200.transformers.models.zafepel import DynamicTanh
    z = SIZES[size]
    W, H, G, D, DH, DG, LH, LD, LV, FF, ROT = (z[k] for k in ("width", "heads", "kv_heads", "dim", "d_heads", "d_kv", "l_heads", "l_dim", "l_vdim", "ff", "rot"))
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
    for phase, B, S, held in (("prefill", 1, PROMPT, 0), ("decode", 8, 1, PROMPT)):
        N, L = B * S, held + S
        pad = torch.zeros(B, dtype=torch.int32, device=dev)
        # the stream
        x, y, yf, wa, step = torch.randn(N, W, device=dev), rnd(N, W), torch.randn(N, W, device=dev), vec(W), vec(W)
        joint = rnd(N, 2 * W)
        add("sum_residual_norms (sum, vector norm)", phase, timer(lambda: ops.sum_residual_norms(x, [y], dtype, 1e-5, gain1=wa)), N * W * (8 + 2 * es))
        add("sum_residual_norms (sum, copy in front of a pass)", phase, timer(lambda: ops.sum_residual_norms(x, [y], dtype, 1e-5, x_copy=joint[:, :W])),
            N * W * (8 + 2 * es))
        add("sum_residual_norms (replaced, pass vector, vector norm)", phase,
            timer(lambda: ops.sum_residual_norms(x, [yf], dtype, 1e-5, gain1=wa, replace=True, vec=step)), N * W * (8 + es))
        post, pre = DynamicTanh(W).to(dtype).to(dev), DynamicTanh(W).to(dtype).to(dev)
        add("dyt_residual_norm", phase, timer(lambda: ops.dyt_residual_norm(x, (y, post), None, pre, dtype)), N * W * (8 + 2 * es),
            like_of="sum_residual_norms")
        # lightning attention
        proj, state = rnd(B, S, LH * (2 * LD + 2 * LV)), torch.zeros(B, LH, LD, LV, device=dev)
        decay = torch.full((LH,), 0.99, device=dev)
        rec = N * (LH * (2 * LD + LV) * es + LH * LV * 4) + 2 * B * LH * LD * LV * 4
        add("constant_decay_attention", phase, timer(lambda: ops.constant_decay_attention(proj, 0, LH, LD, LV, decay, state, held, None)), rec,
            flops=4.0 * N * LH * LD * LV)
        zz = rnd(B, S, LH * LD)
        add("gated_linear_attention", phase, timer(lambda: ops.gated_linear_attention(proj, LH, LD, LV, zz, 16.0, state, held, None)),
            rec + N * LH * LD * es, flops=4.0 * N * LH * LD * LV, like_of="constant_decay_attention")
        o, out = torch.randn(N, LH, LV, device=dev), torch.empty(N, LH * LV, dtype=dtype, device=dev)
        gw, proj2 = vec(LH * LV), proj.view(N, -1)
        off_g = LH * (2 * LD + LV)
        add("gated_rms_norm (all heads together)", phase,
            timer(lambda: ops.gated_rms_norm(o.view(N, 1, LH * LV), proj2, off_g, gw, 1e-5, out, 0, 1.0, sigmoid=True)), N * LH * LV * (4 + 2 * es))
        add("gated_rms_norm (per head, silu)", phase, timer(lambda: ops.gated_rms_norm(o, proj2, off_g, gw[:LV].contiguous(), 1e-5, out, 0, 1.0)),
            N * LH * LV * (4 + 2 * es), like_of="gated_rms_norm (all heads together)")
        # attention branch
        P = 2 * H * D + G * D
        aproj, ks, vs = rnd(B, S, P), rnd(B, G, L, D), rnd(B, G, L, D)
        inv = torch.tensor([500000.0 ** (-2.0 * i / ROT) for i in range(ROT // 2)], dtype=torch.float64, device=dev)
        st = (G * L * D, D, L * D)
        add("rope_qk_prepare (unit-RMS heads, keys as values)", phase,
            timer(lambda: ops.rope_qk_prepare(aproj, 0, H * D, H * D, H, G, D, D, D, 0, 0, ROT, inv, 1.0, ks, st, vs, st, held, 0, pad, eps=1e-5, unit_rms=True)),
            N * (H * D * 2 + G * D * 3) * es)
        qw, kw = vec(D), vec(D)
        q32 = ops.window_qk_prepare(aproj, 0, H * D, H * D + G * D, H, G, D, D, qw, kw, 1e-5, inv, ROT, ks, vs, L, held, 0, pad)
        add("window_qk_prepare", phase,
            timer(lambda: ops.window_qk_prepare(aproj, 0, H * D, H * D + G * D, H, G, D, D, qw, kw, 1e-5, inv, ROT, ks, vs, L, held, 0, pad)),
            N * ((H + 2 * G) * D * es + H * D * 4 + 2 * G * D * es), like_of="rope_qk_prepare")
        q, zero, hb = rnd(N, H * D), torch.zeros(H, dtype=dtype, device=dev), rnd(H)
        wide = torch.empty(N, H * D + DH * D, dtype=dtype, device=dev)
        kview, vview = ks.permute(0, 2, 1, 3), vs.permute(0, 2, 1, 3)
        work = dict(flops=4.0 * D * (S * (S + 1) / 2) * H * B) if S > 1 else dict(bytes_=B * G * L * 2 * D * es)
        add("softmax_attention (a one in the denominator)", phase,
            timer(lambda: ops.softmax_attention(q, kview, vview, B, S, H, held, 0, pad, 0, D ** -0.5, out=wide, sink=zero)), **work)
        add("sigmoid_window_attention (everything visible)", phase,
            timer(lambda: ops.sigmoid_window_attention(q32, ks, vs, L, held, 0, pad, 1 << 20, D ** -0.5, hb, wide, 0, 1.0)),
            like_of="softmax_attention", **work)
        add("sigmoid_gate (channels of a column range)", phase, timer(lambda: ops.sigmoid_gate(wide[:, :H * D], aproj.view(N, P), H * D + G * D, 1, scale=0.7)),
            N * H * D * 3 * es)
        gu = rnd(N, 2 * H * D)
        add("silu_mul", phase, timer(lambda: ops.silu_mul(gu, H * D)), N * H * D * 3 * es, like_of="sigmoid_gate")
        # delta branch
        C = 2 * DG * D + DH * D
        conv, dproj, dz = rnd(B, S, C), rnd(B, S, C + 2 * DH), rnd(B, S, DH * D)
        A_log, dtb_c, dtb_h = rnd(DH) - 1.0, rnd(DH * D), rnd(DH)
        dstate = torch.zeros(B, DH, D, D, device=dev)
        rec = N * (C * es + DH * D * 4) + 2 * B * DH * D * D * 4
        add("channel_delta_rule", phase, timer(lambda: ops.channel_delta_rule(conv, DG, DH, D, D, dproj, C, dz, A_log, dtb_c, dstate, held, None)),
            rec + N * DH * D * es, flops=6.0 * N * DH * D * D)
        add("gated_delta_rule", phase, timer(lambda: ops.gated_delta_rule(conv, DG, DH, D, D, dproj, C, C + DH, A_log, dtb_h, dstate, held, None)),
            rec, flops=6.0 * N * DH * D * D, like_of="channel_delta_rule")
        # feed-forward
        up, coef = rnd(N, FF), vec(4)
        add("gelu_erf", phase, timer(lambda: ops.gelu_erf(up)), N * FF * 2 * es)
        add("poly_norm", phase, timer(lambda: ops.poly_norm(up, coef, 1e-5)), N * FF * 2 * es, like_of="gelu_erf")
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
    out = {"arch": "bugipel", "dtype": "bf16", "data": "synthetic (random weights)",
           "peaks": {"hbm_gbs": peaks["hbm_gbs"], "bf16_tflops": peaks["bf16_tflops"], "source": src},
           "config": {"sizes": SIZES, "layers": LAYERS, "layer_order": ["parallel", "lightning"], "loop": LOOP, "taps": CONV, "vocab": VOCAB,
                      "prompt": PROMPT, "new_tokens": NEW, "cache": "256 MB rewritten between timed runs"}, "kernels": []}
    for size in [s for s in SIZES if not getattr(args, "sizes", None) or s in args.sizes.split(",")]:
        models = [("bugipel_", build_bugipel)] + ([] if args.no_compare else [("zafepel_equal_size_", build_zafepel)])
        for name, build in models:
            model = build(dev, dtype, size)
            out[name + size] = [throughput(model, dev, timer, b) for b in (1, 8)]
            out[name + "recorded_step_failed"] = model.__dict__.get("_b200_state_graph_failed")
            model.__dict__.pop("_b200_state_graphs", None)
            del model
            torch.cuda.empty_cache()
        out["kernels"] += kernel_table(dev, dtype, peaks, timer, size)
    out["zafepel_equal_size_note"] = "bf16, same width / layers / layer runs / heads / recurrent heads / feed-forward width; its window holds everything"
    print(json.dumps(out))
