"""The Bugipel design in the framework against the plain statements of tests/bugipel_oracle.py (float64).

CPU tests cover what needs no kernel: the configuration reader, the order of layer runs, the checkpoint's name map, the merged
projections, the shared output head, the registry, and the oracle's softmax and masks against brute force.  GPU tests run the
kernels (there is no CPU path): every mechanism alone on odd sizes (the constant-decay recurrence in its few-token and pipelined
forms with carried state, the rotation with unit-RMS heads and its cache write, the one in the softmax's denominator in all three
attention kernels, one outstanding key at every place, the channel gate and the norm over all heads, the residual update with
vector norms that replaces the stream and copies it beside the embedding output), then the model: whole prompts against
token-by-token decoding and portions down to two tokens, unequal batches against each request alone, rows leaving a batch, storage
that grows and is used again, long decoding, greedy generation through ``generate()`` and the trace runner's command line.
"""
import json
import os
import subprocess

import pytest
import torch

import bugipel_oracle as O

F64 = torch.float64
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


# ------------------------------------------------------------------ helpers
def save_checkpoint(cfg, weights, folder):
    """config.json + model.safetensors (8-byte header length, JSON header, raw data)"""
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    names = {torch.bfloat16: "BF16", torch.float32: "F32"}
    header, blobs, off = {}, [], 0
    for k, v in weights.items():
        raw = v.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes()
        header[k] = {"dtype": names[v.dtype], "shape": list(v.shape), "data_offsets": [off, off + len(raw)]}
        off += len(raw)
        blobs.append(raw)
    h = json.dumps(header).encode()
    with open(os.path.join(folder, "model.safetensors"), "wb") as f:
        f.write(len(h).to_bytes(8, "little"))
        f.write(h)
        for b in blobs:
            f.write(b)


def load_framework(folder, dtype, device=None, **kw):
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    model = AutoModelForCausalLM.from_pretrained(str(folder), torch_dtype=dtype, **kw)
    return model.to(device) if device is not None else model


def position_errors(got, want):
    """per position: rms over the vocabulary of the difference (mean removed) over the rms of the wanted logits"""
    d = got.to(F64).cpu() - want.to(F64)
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.to(F64).pow(2).mean().sqrt()


def assert_close(got, want, dtype):
    e = position_errors(got, want).reshape(-1)
    if dtype == torch.float32:
        assert e.max() < 3e-5, e.max()
    else:
        assert torch.isfinite(got).all()
        assert e.median() < 0.03 and e.quantile(0.9) < 0.06 and e.max() < 0.2, (e.median(), e.quantile(0.9), e.max())


CONFIGS = {
    # nothing coincides: fewer key than query heads in both branches, dim != vdim, head sizes that are no multiples of 8, a partly
    # rotated head, a layer without feed-forward inside the loop, feed-forwards of different widths, layers before and behind the loop
    "odd": dict(),
    # everything 1 or equal or absent: one head everywhere, one tap, the whole head rotated, scales of 1, no loop
    "plain": dict(width=32, vocab=40, order=("lightning", "parallel"), ffs=(32, None), light=dict(heads=1, dim=8, vdim=8, decay=[0.9]),
                  left=dict(heads=1, kv_heads=1, dim=8, rot_dims=8, scale=1.0), right=dict(heads=1, kv_heads=1, dim=8, vdim=8, conv=1),
                  loop=None, scales=(1.0, 1.0)),
    # head sizes that tile into 16s (the tensor-core attention of a 16-bit model); the loop covers every layer, twice
    "tile": dict(width=64, vocab=83, order=("parallel", "lightning", "parallel"), ffs=(40, None, 72), light=dict(heads=4, dim=32, vdim=64),
                 left=dict(heads=4, kv_heads=2, dim=32, rot_dims=16, base=10000.0, scale=0.2), right=dict(heads=4, kv_heads=1, dim=32, vdim=64, conv=2),
                 loop=(0, 3, 2), scales=(1.2, 0.6)),
    # heads of a served model on a narrow stream: four queries per key head of 128 (decoding takes the kernel that splits the keys of
    # shared heads over blocks), wide recurrent heads, a decay of exactly 1 and one of 0, a loop of one layer that ends the stack
    "wide": dict(width=72, vocab=300, order=("lightning", "lightning", "parallel"), ffs=(100, 24, 64),
                 light=dict(heads=2, dim=136, vdim=24, decay=[1.0, 0.0]), left=dict(heads=8, kv_heads=2, dim=128, rot_dims=32, base=500000.0, scale=0.05),
                 right=dict(heads=2, kv_heads=2, dim=128, vdim=128, conv=4), loop=(2, 3, 4), scales=(0.5, 1.0)),
    # sizes that are multiples of nothing, a loop that runs once, scales of either sign
    "awkward": dict(width=52, vocab=37, order=("parallel", "lightning"), ffs=(25, 11), light=dict(heads=5, dim=3, vdim=7),
                    left=dict(heads=3, kv_heads=3, dim=6, rot_dims=2, base=7.0, scale=-0.3), right=dict(heads=6, kv_heads=3, dim=5, vdim=9, conv=5),
                    loop=(0, 1, 1), scales=(-0.4, 2.0), eps=1e-3),
}
RANKS = {"plain": (1, 1), "awkward": (3, 7), "wide": (16, 8)}


def make(name, seed=0):
    cfg = O.random_config(**CONFIGS[name])
    return cfg, O.random_weights(cfg, seed + 1, ranks=RANKS.get(name, (5, 3)))


def w64(w):
    return {k: v.to(F64) for k, v in w.items()}


def tokens_for(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


# ================================================================== CPU: configuration, loader, order of layers
def test_loader_maps_every_tensor_and_merges(tmp_path):
    cfg, w = make("odd")
    save_checkpoint(cfg, w, tmp_path)
    model = load_framework(tmp_path, torch.bfloat16)
    assert type(model).__name__ == "BugipelForCausalLM" and model.config.model_type == "bugipel"
    assert model.config.low_ranks == {"0": [5, 3], "2": [5, 3]} and model.config.passes == 3
    W = cfg["width"]
    core, layers = model.model, model.model.layers
    assert [l.kind for l in layers] == ["parallel", "lightning", "parallel", "lightning"] and layers[2].mlp is None and not hasattr(layers[2], "norm2")
    assert torch.equal(core.loop_in.weight, w["loop.in"]) and torch.equal(core.loop_step, w["loop.step"]) and core.loop_in.weight.shape == (W, 2 * W)
    assert model.lm_head.weight is core.embed_tokens.weight and torch.equal(model.lm_head.weight, w["embed"])
    li = layers[1].mixer                                                    # q, k: 3 x 10; v, gate: 3 x 14
    assert li.in_proj.weight.shape == (60 + 84, W) and not hasattr(li, "q_proj") and li.norm.weight.shape == (42,)
    assert torch.equal(li.in_proj.weight[30:60], w["l1.mix.k"]) and torch.equal(li.in_proj.weight[102:], w["l1.mix.g"])
    assert li.decay.on(torch.device("cpu")).tolist() == pytest.approx(cfg["layers"][1]["mixer"]["decay"])
    pm = layers[0].mixer                                                    # left 72 + 24 + 72; right 12 + 12 + 40 + 4 + 5 + 3
    assert pm.in_proj.weight.shape == (168 + 76, W) and pm.out_proj.weight.shape == (W, 72 + 40)
    assert torch.equal(pm.in_proj.weight[72:96], w["l0.mix.left.k"]) and torch.equal(pm.in_proj.weight[96:168], w["l0.mix.left.g"])
    assert torch.equal(pm.in_proj.weight[236:241], w["l0.mix.right.a1"]) and torch.equal(pm.out_proj.weight[:, 72:], w["l0.mix.right.o"])
    assert pm.right.in_columns == 76 and torch.equal(pm.right.conv_weight[12:24], w["l0.mix.right.k.conv"])
    assert (pm.left_scale, pm.right_scale, pm.left.rotary.dims, pm.left.scale) == (0.7, 1.3, 8, 0.4)
    assert torch.equal(layers[3].mlp.up_proj.weight, w["l3.mlp.up"]) and layers[3].mlp.up_proj.out_features == 33
    # a missing tensor and a tensor of the wrong shape are refused, by name
    for name, bad in (("l2.mix.right.g2", None), ("l0.mix.right.dt_bias", torch.zeros(4, dtype=torch.bfloat16)), ("loop.step", torch.zeros(2, W).bfloat16())):
        broken = dict(w)
        if bad is None:
            del broken[name]
        else:
            broken[name] = bad
        save_checkpoint(cfg, broken, tmp_path / "bad")
        with pytest.raises(RuntimeError, match=name.split(".")[-1]):
            load_framework(tmp_path / "bad", torch.bfloat16)


def test_unsupported_configurations_are_refused(tmp_path):
    for change, text in ((lambda c: c["layers"][0]["mixer"]["left"].update(vdim=6), "vdim"), (lambda c: c["layers"][1]["mixer"].update(decay=[0.5]), "decay"),
                         (lambda c: c["layers"][1].update(type="other"), "layer type"), (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "feed-forward")):
        cfg, w = make("odd")
        change(cfg)
        save_checkpoint(cfg, w, tmp_path)
        with pytest.raises(RuntimeError, match=text):
            load_framework(tmp_path, torch.bfloat16)


def test_registry_picks_the_design(tmp_path):
    from ipex_llm_b200.transformers.model import native_architecture
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Bugipel"}))
    assert native_architecture(tmp_path).endswith("models.bugipel")


def test_order_of_layer_runs():
    from ipex_llm_b200.transformers.models.bugipel import BugipelConfig
    layers = [{"type": "lightning"}] * 4
    assert BugipelConfig(layers=layers).layer_runs() == [(0, None), (1, None), (2, None), (3, None)]
    got = BugipelConfig(layers=layers, loop={"start": 1, "stop": 3, "times": 2}).layer_runs()
    assert got == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert BugipelConfig(layers=layers, loop={"start": 3, "stop": 4, "times": 3}).layer_runs() == [(0, None), (1, None), (2, None), (3, 0), (3, 1), (3, 2)]
    assert BugipelConfig(layers=layers, loop={"start": 0, "stop": 4, "times": 1}).layer_runs() == [(0, 0), (1, None), (2, None), (3, None)]
    for loop in (None, (1, 3, 2), (0, 4, 1), (3, 4, 3)):
        cfg = {"layers": layers, "loop": loop and {"start": loop[0], "stop": loop[1], "times": loop[2]}}
        assert O.layer_runs(cfg) == BugipelConfig(**cfg).layer_runs()
    with pytest.raises(RuntimeError):
        BugipelConfig(layers=layers, loop={"start": 2, "stop": 5, "times": 2}).layer_runs()


def test_oracle_softmax_with_a_one_in_the_denominator():
    s = torch.tensor([[0.0, 1.0, -2.0], [300.0, 299.0, 0.0], [-300.0, -301.0, -400.0]], dtype=F64)
    p = O.softmax_with_one(s)
    e = torch.exp(s[0])
    assert torch.allclose(p[0], e / (1 + e.sum())) and p[0].sum() < 0.9
    assert torch.allclose(p[1], torch.softmax(s[1], 0)) and p[2].sum() < 1e-100 and torch.isfinite(p).all()


# ================================================================== GPU: each mechanism alone
@pytest.fixture(scope="module")
def mixers(cuda_device):
    from ipex_llm_b200.transformers.models import mixer_ops
    return mixer_ops


def _rand(shape, gen, dtype, device, scale=1.0):
    return (torch.randn(shape, generator=gen) * scale).to(dtype).to(device)


def _c64(t):
    return t.cpu().to(F64)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("H,D,Dv,sizes", [(4, 12, 10, (70, 1, 5)), (2, 136, 24, (20, 3)), (3, 32, 64, (1, 1, 33, 2)), (1, 8, 8, (4, 4)),
                                          (3, 48, 32, (129,)), (40, 64, 64, (36, 20)), (2, 520, 8, (18, 2)), (5, 3, 200, (17, 16, 15))])
def test_constant_decay_attention_with_carried_state(mixers, cuda_device, dtype, H, D, Dv, sizes):
    """the few-token and the pipelined kernel, the state carried from call to call, a row whose first tokens are padding, columns out
    of the middle of a wider projection; decays from 0 (only the token itself) to 1 (nothing is forgotten)"""
    g = torch.Generator().manual_seed(H * D + Dv)
    B, T, off = 2, sum(sizes), 3
    pads = [0, min(3, sizes[0] - 1)]
    proj = _rand((B, T, off + H * (2 * D + Dv) + 2), g, dtype, cuda_device)
    decay = torch.linspace(0.0, 1.0, H + 1)[1:] if H > 1 else torch.tensor([0.83])
    decay[0] = 0.0 if H > 2 else decay[0]
    state = torch.zeros(B, H, D, Dv, dtype=torch.float32, device=cuda_device)
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    for silu in (True, False):
        state.zero_()
        out, at = [], 0
        for n in sizes:
            out.append(mixers.constant_decay_attention(proj[:, at:at + n].contiguous(), off, H, D, Dv, decay.to(cuda_device), state, at,
                                                       pad if at == 0 else None, silu=silu))
            at += n
        got = _c64(torch.cat(out, dim=1))
        for b, p in enumerate(pads):
            c = _c64(proj[b, p:, off:off + H * (2 * D + Dv)])
            c = O.silu(c) if silu else c
            n = T - p
            want = O.constant_decay_scan(c[:, :H * D].view(n, H, D), c[:, H * D:2 * H * D].view(n, H, D), c[:, 2 * H * D:].view(n, H, Dv), decay.to(F64))
            assert ((got[b, p:] - want).abs() / (want.abs().max() + 1)).max() < 3e-6, (silu, b)       # inputs are exact, the rest is 32-bit
            assert got[b, :p].abs().sum() == 0
    assert (O.silu(c) - c).abs().max() > 0.1


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("held,shift", [(0, 0), (6, 4000)])
@pytest.mark.parametrize("H,G,D,dims", [(6, 2, 12, 8), (3, 3, 10, 10), (4, 1, 64, 0), (2, 2, 130, 128)])
def test_rotation_then_unit_rms_and_the_raw_keys_as_values(mixers, cuda_device, dtype, held, shift, H, G, D, dims):
    """queries and keys rotated and divided by their root mean square, values stored as the keys come in; far positions keep their
    angle, padding slots hold zeros, neighbours in the cache stay untouched"""
    g = torch.Generator().manual_seed(D)
    B, S, cap, eps = 2, 5, 16, 0.05                                          # an eps that matters
    pads = [0, 2]
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    tol = 2e-5 if dtype == torch.float32 else 0.02
    base, off_k = 50.0, H * D + 1
    inv = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)] or [0.0], dtype=F64, device=cuda_device)
    proj = _rand((B, S, off_k + G * D + 3), g, dtype, cuda_device, 0.5)
    ks, vs = torch.full((B, G, cap, D), 9.0, dtype=dtype, device=cuda_device), torch.full((B, G, cap, D), 9.0, dtype=dtype, device=cuda_device)
    st = (G * cap * D, D, cap * D)
    q = mixers.rope_qk_prepare(proj, 0, off_k, off_k, H, G, D, D, D, 0, 0, dims, inv, 1.0, ks, st, vs, st, held, shift, pad, eps=eps, unit_rms=True)
    for b in range(B):
        first = max(pads[b] - held - shift, 0)
        pos = torch.arange(S) + held + shift - pads[b]
        raw_k = _c64(proj[b, :, off_k:off_k + G * D]).view(S, G, D)
        want_q, want_k = O.prepare_qk(_c64(proj[b, :, :H * D]).view(S, H, D), raw_k, pos, {"dims": dims, "base": base}, eps)
        assert (_c64(q.view(B, S, H, D)[b, first:]) - want_q[first:]).abs().max() < tol
        assert (_c64(ks[b, :, held + first:held + S]).transpose(0, 1) - want_k[first:]).abs().max() < tol
        assert torch.equal(_c64(vs[b, :, held + first:held + S]).transpose(0, 1), raw_k[first:])
        assert ks[b, :, held:held + first].abs().sum() == 0 and vs[b, :, held:held + first].abs().sum() == 0
        for t in (ks, vs):
            assert (t[b, :, :held] == 9).all() and (t[b, :, held + S:] == 9).all()
    assert (want_k - raw_k).abs().max() > 0.1


ATTENTION = [(torch.float32, 5, 0, 6, 2, 5, 7, False), (torch.float32, 1, 300, 4, 1, 24, 40, False), (torch.bfloat16, 1, 517, 3, 1, 64, 64, False),
             (torch.bfloat16, 40, 30, 4, 2, 32, 16, True), (torch.float16, 150, 0, 3, 1, 64, 48, True), (torch.bfloat16, 1, 700, 8, 2, 128, 128, True),
             (torch.bfloat16, 3, 130, 4, 1, 32, 256, True)]


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,S,held,H,G,D,Dv,tc", ATTENTION)
def test_a_one_in_the_denominator_in_every_attention_kernel(mixers, cuda_device, dtype, S, held, H, G, D, Dv, tc):
    """the general kernel, the prompt kernel on the tensor cores and the split-key kernel with a sink of score 0, written into the
    middle of a wider buffer: scores around zero (the one takes a visible share), far below zero (the one takes everything) and far
    above (the one vanishes)"""
    g = torch.Generator().manual_seed(S + held)
    B, L = 2, held + S
    k, v = _rand((B, L + 3, G, D + 8), g, dtype, cuda_device)[..., 8:], _rand((B, L + 3, G, Dv + 16), g, dtype, cuda_device)[..., :Dv]
    pads = [0, min(L - 1, 3)]
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    zero = torch.zeros(H, dtype=dtype, device=cuda_device)
    tol = 2e-5 if dtype == torch.float32 else 0.02
    for lift, scale in ((0.0, 0.3 / D ** 0.5), (-6.0, 1.0), (4.0, 1.0)):
        q = _rand((B * S, H * D), g, dtype, cuda_device, 0.2)
        kk = k.clone()
        if lift:                                                            # one channel that shifts every score by the same amount
            q = q.view(B * S, H, D).clone()
            q[..., 0], kk[..., 0] = 4.0, lift
            q = q.view(B * S, H * D)
        out = torch.full((B * S, H * Dv + 24), 7.0, dtype=dtype, device=cuda_device)
        mixers.softmax_attention(q, kk, v, B, S, H, held, 0, pad, 0, scale, out=out, out_col=8, tensor_cores=tc, sink=zero)
        assert (out[:, :8] == 7).all() and (out[:, 8 + H * Dv:] == 7).all()
        got = out[:, 8:8 + H * Dv].reshape(B, S, H, Dv)
        for b in range(B):
            args = (_c64(q.view(B, S, H, D)[b]), _c64(kk[b]), _c64(v[b]), scale, held, pads[b])
            want, without = O.visible_attention(*args), O.visible_attention(*args, sink=False)
            assert (_c64(got[b]) - want).abs().max() < tol, (lift, b)
            if lift < 0:
                assert want.abs().max() < 0.02 and without[-1].abs().max() > 0.05
    # the first token of a sequence sees itself and the one: p = e^s / (1 + e^s)
    q = _rand((1, H * D), g, dtype, cuda_device)
    one = mixers.softmax_attention(q, k[:1, :1], v[:1, :1], 1, 1, H, 0, 0, pad[:1], 0, 0.1, tensor_cores=tc, sink=zero)
    s = torch.einsum("hd,hd->h", _c64(q).view(H, D), _c64(k[0, 0]).repeat_interleave(H // G, 0)) * 0.1
    want = torch.sigmoid(s)[:, None] * _c64(v[0, 0]).repeat_interleave(H // G, 0)
    assert (_c64(one).view(H, Dv) - want).abs().max() < tol


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,S,tc", [(torch.float32, 1, False), (torch.float32, 40, False), (torch.bfloat16, 1, False), (torch.bfloat16, 40, True),
                                        (torch.bfloat16, 1, True), (torch.bfloat16, 9, True)])
def test_one_outstanding_key_anywhere(mixers, cuda_device, dtype, S, tc):
    """a key whose score dwarfs all others (and the sink): its value is the output wherever it sits -- the first token, the borders of
    the kernels' key tiles, far back, the query itself -- and it must not show from the future or from in front of the row's first
    token, for the last of the new tokens and for one in their middle"""
    g = torch.Generator().manual_seed(11)
    H, D, Dv, L = 4, 16, 128, 1300
    held = L - S
    base_k, base_v = torch.randn(1, L + 8, 1, D, generator=g) * 0.1, torch.randn(1, L + 8, 1, Dv, generator=g)
    spike = torch.zeros(D)
    spike[3] = 40.0
    q = (torch.randn(S, H * D, generator=g) * 0.1 + spike.repeat(H)[None] * 0.05).to(dtype).to(cuda_device)
    v_dev, zero = base_v.to(dtype).to(cuda_device), torch.zeros(H, dtype=dtype, device=cuda_device)

    def shows(at, query=S - 1, first=0):
        k = base_k.clone()
        k[0, at, 0] = spike
        out = mixers.softmax_attention(q, k.to(dtype).to(cuda_device), v_dev, 1, S, H, held, 0, torch.tensor([first], dtype=torch.int32, device=cuda_device),
                                       0, 1.0, tensor_cores=tc, sink=zero)
        d = (out.float().cpu().view(S, H, Dv)[query] - base_v[0, at, 0]).abs().max()
        assert d < 0.03 or d > 0.3, d
        return bool(d < 0.03)

    for at in (0, 1, 31, 32, 63, 64, 255, 256, 257, 511, 512, 1023, 1024, L - 2, L - 1):
        assert shows(at), at
    assert not shows(L) and not shows(4, first=5) and shows(5, first=5)
    if S > 21:
        assert shows(held + 20, query=20) and not shows(held + 21, query=20) and shows(held + 21, query=21)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_channel_gate_in_a_column_range_and_the_norm_over_all_heads(mixers, cuda_device, dtype):
    g = torch.Generator().manual_seed(2)
    eps = 1e-3
    tol = 1e-5 if dtype == torch.float32 else 0.04
    n, C = 9, 70
    buf = _rand((n, C + 30), g, dtype, cuda_device)
    gate = _rand((n, 3 + C + 2), g, dtype, cuda_device, 2.0)
    before = buf.clone()
    mixers.sigmoid_gate(buf[:, 10:10 + C], gate, 3, 1, scale=-0.7)
    assert torch.equal(buf[:, :10], before[:, :10]) and torch.equal(buf[:, 10 + C:], before[:, 10 + C:])
    assert (_c64(buf[:, 10:10 + C]) + 0.7 * _c64(before[:, 10:10 + C]) * torch.sigmoid(_c64(gate[:, 3:3 + C]))).abs().max() < tol
    # one root mean square over all heads together (rows of 42 to 2600 channels, a few rows and many)
    for n, H, Dv in ((7, 3, 14), (5, 4, 300), (1500, 2, 200), (2, 13, 200), (1300, 8, 256)):
        o = torch.randn(n, H, Dv, generator=g)
        o *= torch.arange(1, H + 1).view(1, H, 1)                           # heads of different size: a norm per head would show
        o = o.to(cuda_device)
        gate, w = _rand((n, H * Dv + 4), g, dtype, cuda_device), _rand((H * Dv,), g, dtype, cuda_device) + 1.0
        out = torch.empty(n, H * Dv, dtype=dtype, device=cuda_device)
        mixers.gated_rms_norm(o.view(n, 1, H * Dv), gate, 4, w, eps, out, 0, 1.0, sigmoid=True)
        flat = _c64(o).reshape(n, H * Dv)
        want = O.unit_rms(flat, eps) * _c64(w) * torch.sigmoid(_c64(gate[:, 4:]))
        assert ((_c64(out) - want).abs() / (1 + want.abs())).max() < tol
        per_head = O.unit_rms(_c64(o), eps).reshape(n, H * Dv) * _c64(w) * torch.sigmoid(_c64(gate[:, 4:]))
        assert (per_head - want).abs().max() > 0.1


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,n", [(45, 5), (1100, 3), (352, 1500), (8200, 2), (2000, 70), (1, 4)])
def test_residual_update_with_vector_norms(mixers, cuda_device, dtype, width, n):
    """x += y, a norm with one weight per channel, a copy of the new stream beside the embedding output; and a pass's entry: the
    stream replaced by a 32-bit projection plus the pass's vector -- rows in registers and the plain loop"""
    g = torch.Generator().manual_seed(width)
    eps = 1e-3
    tol = 3e-5 if dtype == torch.float32 else 0.05
    x0 = torch.randn(n, width, generator=g) * 2 + 0.5
    y, yf = _rand((n, width), g, dtype, cuda_device), _rand((n, width), g, torch.float32, cuda_device)
    w1, w2, vec = (_rand((width,), g, dtype, cuda_device, 0.4) + 1.0 for _ in range(3))
    joint = torch.full((n, 2 * width), 7.0, dtype=dtype, device=cuda_device)
    x = x0.clone().to(cuda_device)
    h1, h2 = mixers.sum_residual_norms(x, [y], dtype, eps, gain1=w1, gain2=w2, x_copy=joint[:, :width])
    new = x0.to(F64) + _c64(y)
    assert (_c64(x) - new).abs().max() < 1e-5 and (_c64(joint[:, :width]) - new).abs().max() < tol and (joint[:, width:] == 7).all()
    assert ((_c64(h1) - O.unit_rms(new, eps) * _c64(w1)).abs()).max() < tol and (_c64(h2) - O.unit_rms(new, eps) * _c64(w2)).abs().max() < tol
    # only the copy is wanted (what precedes a pass)
    x = x0.clone().to(cuda_device)
    assert mixers.sum_residual_norms(x, [y], dtype, eps, x_copy=joint[:, width:]) == (None, None)
    assert (_c64(joint[:, width:]) - new).abs().max() < tol and (_c64(x) - new).abs().max() < 1e-5
    # replaced, plus a vector; what x held does not matter, not even infinities
    x.fill_(float("inf"))
    h1, none = mixers.sum_residual_norms(x, [yf], dtype, eps, gain1=w1, replace=True, vec=vec)
    new = _c64(yf) + _c64(vec)
    assert none is None and (_c64(x) - new).abs().max() < 1e-5 and (_c64(h1) - O.unit_rms(new, eps) * _c64(w1)).abs().max() < tol


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_projection_into_32_bit(cuda_device, dtype):
    """a 16-bit projection answers with its 32-bit accumulator: no rounding behind the product"""
    from ipex_llm_b200.transformers.models.mixers import linear_f32
    g = torch.Generator().manual_seed(1)
    lin = torch.nn.Linear(96, 40, bias=False)
    lin.weight = torch.nn.Parameter(_rand((40, 96), g, dtype, cuda_device), requires_grad=False)
    x = _rand((7, 96), g, dtype, cuda_device)
    got = linear_f32(lin, x)
    assert got.dtype == torch.float32 and (_c64(got) - _c64(x) @ _c64(lin.weight).T).abs().max() < 1e-4


# ================================================================== GPU: the model
def build(tmp_path, name, dtype, device, seed=0, **kw):
    cfg, w = make(name, seed)
    folder = tmp_path / f"{name}{seed}"
    save_checkpoint(cfg, w, folder)
    return cfg, w64(w), load_framework(folder, dtype, device, **kw)


@torch.no_grad()
def run_portions(model, tokens, sizes, device):
    """one request fed in portions (the last size repeats); returns logits [T, V]"""
    ids = torch.tensor([tokens], device=device)
    cache, out, at, i = None, [], 0, 0
    while at < len(tokens):
        n = sizes[min(i, len(sizes) - 1)]
        o = model(input_ids=ids[:, at:at + n], past_key_values=cache, use_cache=True)
        cache = o.past_key_values
        out.append(o.logits[0])
        at, i = at + n, i + 1
    return torch.cat(out)


@pytest.mark.gpu
@pytest.mark.parametrize("name", list(CONFIGS))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_whole_decode_and_portions_against_the_oracle(tmp_path, cuda_device, name, dtype):
    cfg, w, model = build(tmp_path, name, dtype, cuda_device)
    tokens = tokens_for(cfg, 200 if name == "wide" else 75, 3)
    collect = []
    want = O.forward(cfg, w, tokens, collect)
    model.collect_residual = []
    whole = run_portions(model, tokens, [len(tokens)], cuda_device)
    assert len(model.collect_residual) == len(collect) == len(O.layer_runs(cfg))
    if dtype == torch.float32:                                              # the stream after every layer run, too
        for got, ref in zip(model.collect_residual, collect):
            assert (got[0].cpu().to(F64) - ref).abs().max() < 1e-4 * max(1.0, ref.abs().max())
    model.collect_residual = None
    assert_close(whole, want, dtype)
    assert_close(run_portions(model, tokens, [40, 1], cuda_device), want, dtype)                   # a prompt, then token by token
    assert_close(run_portions(model, tokens, [1], cuda_device), want, dtype)                       # from the first token on
    for sizes in ([2], [3, 17, 2, 30], [20, 20, 19, 16], [1, 1, 40, 2]):
        assert_close(run_portions(model, tokens, sizes, cuda_device), want, dtype)
    if dtype != torch.float32:                                              # the general attention kernel under a 16-bit model
        model.attention_tensor_cores = False
        assert_close(run_portions(model, tokens, [len(tokens)], cuda_device), want, dtype)
    # the kept positions may be chosen
    ids = torch.tensor([tokens], device=cuda_device)
    with torch.no_grad():
        some = model(input_ids=ids, logits_to_keep=torch.tensor([0, 7, 30])).logits[0]
        last = model(input_ids=ids, logits_to_keep=2).logits[0]
    assert_close(some, want[[0, 7, 30]], dtype)
    assert_close(last, want[-2:], dtype)


@pytest.mark.gpu
def test_every_branch_shows_in_the_logits(tmp_path, cuda_device):
    """leaving out or changing one mechanism in the plain statement moves the logits far more than the framework differs from it"""
    cfg, w, model = build(tmp_path, "odd", torch.float32, cuda_device)
    tokens = tokens_for(cfg, 40, 3)
    got = run_portions(model, tokens, [25, 1], cuda_device)

    def moved(change_w=None, change_cfg=None, **patch):
        c2, w2 = json.loads(json.dumps(cfg)), dict(w)
        if change_cfg:
            change_cfg(c2)
        if change_w:
            change_w(w2)
        saved = {k: getattr(O, k) for k in patch}
        try:
            for k, v in patch.items():
                setattr(O, k, v)
            return position_errors(got, O.forward(c2, w2, tokens)).max().item()
        finally:
            for k, v in saved.items():
                setattr(O, k, v)

    assert moved() < 3e-5
    assert moved(softmax_with_one=lambda s: torch.softmax(s, -1)) > 1e-3                                 # the sink left out
    unrotated = lambda q, k, p, rot, eps: (O.unit_rms(q, eps), O.unit_rms(k, eps))                       # noqa: E731
    assert moved(prepare_qk=unrotated) > 1e-3
    unnormed = lambda q, k, p, rot, eps: (O.rotate_half(q, p, rot["dims"], rot["base"]), O.rotate_half(k, p, rot["dims"], rot["base"]))    # noqa: E731
    assert moved(prepare_qk=unnormed) > 1e-3
    assert moved(enter_pass=lambda x, x0, wt, t: torch.cat([x, x0], -1) @ wt["loop.in"].T + wt["loop.step"][0]) > 1e-3
    assert moved(enter_pass=lambda x, x0, wt, t: torch.cat([x0, x], -1) @ wt["loop.in"].T + wt["loop.step"][t]) > 1e-3
    assert moved(enter_pass=lambda x, x0, wt, t: x + wt["loop.step"][t]) > 1e-3
    assert moved(change_cfg=lambda c: c["layers"][1]["mixer"]["decay"].reverse()) > 1e-3
    assert moved(change_cfg=lambda c: c["layers"][0]["mixer"].update(left_scale=1.0)) > 1e-3
    assert moved(change_cfg=lambda c: c["loop"].update(times=2)) > 1e-3
    assert moved(change_w=lambda x: x.update({"l0.mix.right.q.conv": torch.flip(x["l0.mix.right.q.conv"], [1])})) > 1e-3
    assert moved(gelu_erf=lambda z: 0.5 * z * (1 + torch.tanh(0.7978845608 * (z + 0.044715 * z ** 3)))) > 1e-4


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["odd", "tile", "plain", "wide"])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_unequal_batch_matches_each_request_alone(tmp_path, cuda_device, name, dtype):
    cfg, w, model = build(tmp_path, name, dtype, cuda_device)
    lens, extra = [1, 23, 50, 7], 12
    seqs = [tokens_for(cfg, n + extra, 20 + n) for n in lens]
    want = [O.forward(cfg, w, s) for s in seqs]
    width = max(lens)
    ids = torch.zeros(4, width, dtype=torch.int64)
    mask = torch.zeros(4, width, dtype=torch.int64)
    for b, (s, n) in enumerate(zip(seqs, lens)):
        ids[b, width - n:] = torch.tensor(s[:n])
        mask[b, width - n:] = 1
    with torch.no_grad():
        o = model(input_ids=ids.to(cuda_device), attention_mask=mask.to(cuda_device), use_cache=True)
        cache = o.past_key_values
        got = [[o.logits[b, width - n:]] for b, n in enumerate(lens)]
        rows = [0, 1, 2, 3]
        for step in range(extra):
            if step == 2:                                                   # two requests end: their rows leave the batch
                cache.batch_select_indices(torch.tensor([3, 1]))
                rows = [3, 1]
            nxt = torch.tensor([[seqs[b][lens[b] + step]] for b in rows], device=cuda_device)
            o = model(input_ids=nxt, past_key_values=cache, use_cache=True)
            for r, b in enumerate(rows):
                got[b].append(o.logits[r])
    for b in range(4):
        g = torch.cat(got[b])
        assert_close(g, want[b][:g.shape[0]], dtype)


@pytest.mark.gpu
def test_long_decoding(tmp_path, cuda_device):
    """300 tokens one by one from a 5-token prompt: the stores of both passes outgrow their first block and move, the recurrent states
    and the tails are carried 300 times; the same request in portions around the store's block size"""
    cfg, w, model = build(tmp_path, "tile", torch.float32, cuda_device)
    tokens = tokens_for(cfg, 305, 9)
    want = O.forward(cfg, w, tokens)
    assert_close(run_portions(model, tokens, [5, 1], cuda_device), want, torch.float32)
    for sizes in ([255, 2, 48], [256, 1, 1, 47], [257, 48], [15, 16, 17, 2]):
        assert_close(run_portions(model, tokens, sizes, cuda_device), want, torch.float32)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["attention", "lightning", "delta"])
def test_a_far_token_reaches_the_last_logits(tmp_path, cuda_device, kind):
    """changing one early token of a long prompt changes the last position's logits exactly as the plain statement says, in a prompt and
    when the tail is decoded token by token, through each mixer alone (a parallel layer's other branch is scaled away): the attention
    sees everything, the recurrences' states hardly decay"""
    spec = dict(CONFIGS["odd"], ffs=(None,) * 4)
    if kind == "lightning":
        spec.update(order=("lightning",), ffs=(None,), light=dict(heads=2, dim=10, vdim=14, decay=[0.9999, 1.0]), loop=None)
    else:
        spec.update(order=("parallel",), ffs=(None,), loop=(0, 1, 2), scales=(1.0, 0.0) if kind == "attention" else (0.0, 1.0),
                    left=dict(heads=4, kv_heads=2, dim=8, rot_dims=2, base=1e9, scale=1.5))
    cfg = O.random_config(**spec)
    w = O.random_weights(cfg, 5)
    for k in w:
        if k.endswith("A_log"):
            w[k] = w[k] - 6.0
    folder = tmp_path / kind
    save_checkpoint(cfg, w, folder)
    w, model = w64(w), load_framework(folder, torch.float32, cuda_device)
    tokens = tokens_for(cfg, 260, 13)
    for at in (0, 1, 37):
        other = list(tokens)
        other[at] = (other[at] + 1) % cfg["vocab"]
        want_a, want_b = O.forward(cfg, w, tokens)[-1:], O.forward(cfg, w, other)[-1:]
        assert position_errors(want_a, want_b).max() > 3e-4                 # the early token matters
        for sizes in ([260], [200, 1], [2, 258]):
            assert position_errors(run_portions(model, other, sizes, cuda_device)[-1:], want_b).max() < 2e-5


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["odd", "plain", "tile"])
def test_greedy_generate_matches_the_oracle(tmp_path, cuda_device, name):
    cfg, w, model = build(tmp_path, name, torch.float32, cuda_device)
    prompt = tokens_for(cfg, 9, 4)
    want = O.greedy(cfg, w, prompt, 12)
    ids = torch.tensor([prompt], device=cuda_device)
    got = model.generate(ids, max_new_tokens=12, do_sample=False)
    assert model.__dict__.get("_b200_state_graph_failed") is None and model.__dict__.get("_b200_state_graphs")     # the recorded step ran
    assert got[0].tolist() == want
    # the step's cache serves other requests afterwards: a batch of two with padding, then the first request again
    other = tokens_for(cfg, 4, 5)
    want2 = O.greedy(cfg, w, other, 7)
    batch = torch.tensor([prompt, [0] * 5 + other], device=cuda_device)
    mask = torch.tensor([[1] * 9, [0] * 5 + [1] * 4], device=cuda_device)
    got2 = model.generate(batch, attention_mask=mask, max_new_tokens=7, do_sample=False)
    assert got2[0].tolist() == want[:16] and got2[1, 5:].tolist() == want2
    assert model.generate(ids, max_new_tokens=12, do_sample=False)[0].tolist() == want
    # sampling goes through transformers' loop on the same forward
    torch.manual_seed(0)
    sampled = model.generate(ids, max_new_tokens=5, do_sample=True, top_k=3)
    assert sampled.shape == (1, 14) and sampled[0, :9].tolist() == prompt


@pytest.mark.gpu
def test_recorded_step_of_a_16_bit_model_equals_the_eager_loop(tmp_path, cuda_device, monkeypatch):
    """a bf16 model whose attention decodes through the kernel that splits the keys of shared heads over blocks: the replayed step
    reads the cache length from the device and must produce the tokens of the loop that passes it from the host; every pass's
    states and tails are updated in place by both; the prompts take the tensor-core attention and (padded) two streams"""
    cfg, w, model = build(tmp_path, "wide", torch.bfloat16, cuda_device)
    from ipex_llm_b200.ggml.model import mixers_cpp
    assert mixers_cpp.lib().mixers_softmax_attention_workspace(mixers_cpp.dtype_code(torch.bfloat16), 2, 1, 8, 2, 128, 128) > 0
    prompts = torch.tensor([tokens_for(cfg, 150, 1), [0] * 30 + tokens_for(cfg, 120, 2)], device=cuda_device)
    mask = torch.tensor([[1] * 150, [0] * 30 + [1] * 120], device=cuda_device)
    replayed = model.generate(prompts, attention_mask=mask, max_new_tokens=80, do_sample=False)
    assert model.__dict__.get("_b200_state_graph_failed") is None and model.__dict__.get("_b200_state_graphs")
    monkeypatch.setenv("IPEX_LLM_B200_DECODE_GRAPH", "0")
    eager = model.generate(prompts, attention_mask=mask, max_new_tokens=80, do_sample=False)
    assert torch.equal(replayed, eager)
    for b, n in ((0, 150), (1, 120)):                                       # and both follow the plain statement where it is no close call
        want = O.forward(cfg, w, prompts[b, 150 - n:].tolist())[-1]
        top2 = want.topk(2).values
        if top2[0] - top2[1] > 0.2 * want.std():
            assert int(replayed[b, 150]) == int(want.argmax())


@pytest.mark.gpu
def test_low_bit_conversion_runs_the_same_model(tmp_path, cuda_device, native_lib):
    """the projections are ordinary linears to the converter: a sym_int4 model answers close to the 16-bit one; the head becomes a
    low-bit copy while the embedding table keeps its type; saved and loaded again it gives the same logits"""
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    from ipex_llm_b200.transformers.low_bit_linear import LowBitLinear
    cfg = O.random_config(width=128, vocab=90, order=("parallel", "lightning"), ffs=(192, 64), light=dict(heads=2, dim=32, vdim=64),
                          left=dict(heads=4, kv_heads=2, dim=32, rot_dims=32), right=dict(heads=2, kv_heads=1, dim=32, vdim=64), loop=(0, 2, 2))
    w = O.random_weights(cfg, 3, ranks=(64, 64))
    save_checkpoint(cfg, w, tmp_path / "m")
    ref = load_framework(tmp_path / "m", torch.bfloat16, cuda_device)
    low = load_framework(tmp_path / "m", torch.bfloat16, None, load_in_low_bit="sym_int4").to(cuda_device)
    pm = low.model.layers[0].mixer
    assert all(isinstance(m, LowBitLinear) for m in (pm.in_proj, pm.out_proj, pm.right.a2_proj, low.model.loop_in, low.lm_head, low.model.layers[1].mlp.down_proj))
    assert low.model.embed_tokens.weight.dtype == torch.bfloat16
    tokens = tokens_for(cfg, 30, 1)
    a = run_portions(ref, tokens, [30], cuda_device)
    b = run_portions(low, tokens, [25, 1], cuda_device)
    assert torch.isfinite(b).all() and position_errors(b, a.cpu().to(F64)).quantile(0.8) < 0.5
    low.save_low_bit(str(tmp_path / "low"))
    back = AutoModelForCausalLM.load_low_bit(str(tmp_path / "low")).to(cuda_device)
    again = run_portions(back, tokens, [25, 1], cuda_device)
    assert position_errors(again, b.cpu().to(F64)).max() < 0.02


@pytest.mark.gpu
def test_trace_runner_replays_batches_and_gives_rows_back(tmp_path, cuda_device):
    """the command line a user replays a trace with: requests of unequal length start together and are decoded together, one ends
    early, a second batch starts afterwards (its rows take the place the first batch gave back); float32, against the plain
    statement position by position"""
    cfg, w = make("odd")
    save_checkpoint(cfg, w, tmp_path / "m")
    seqs = {"a": tokens_for(cfg, 31, 1), "b": tokens_for(cfg, 12, 2), "c": tokens_for(cfg, 20, 3), "d": tokens_for(cfg, 9, 4)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seqs["a"][:25], "want": [0, 24]}, {"id": "b", "tokens": seqs["b"][:6], "want": [5]}], "end": []}]
    for i in range(6):                                                      # b ends behind step 4, a goes on alone
        want = [] if i == 2 else [0]
        entries = [{"id": "a", "tokens": [seqs["a"][25 + i]], "want": want}, {"id": "b", "tokens": [seqs["b"][6 + i]], "want": want}]
        steps.append({"step": 1 + i, "entries": entries[:2 if i < 4 else 1], "end": ["b"] if i == 3 else []})   # step 3 wants nothing: no file
    steps.append({"step": 7, "entries": [{"id": "c", "tokens": seqs["c"], "want": [19]}, {"id": "d", "tokens": seqs["d"], "want": [0, 8]}], "end": ["a", "c", "d"]})
    out = tmp_path / "out"
    env = dict(os.environ, PYTHONPATH=ROOT + os.pathsep + os.environ.get("PYTHONPATH", ""))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out", str(out), "--max-tokens", "64"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, env=env, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(8)]
    full = {k: O.forward(cfg, w64(w), s) for k, s in seqs.items()}
    V = cfg["vocab"]

    def rows(step):
        return torch.frombuffer(bytearray((out / f"{step}.f32").read_bytes()), dtype=torch.float32).view(-1, V)

    assert not (out / "3.f32").exists()
    assert_close(rows(0), torch.stack([full["a"][0], full["a"][24], full["b"][5]]), torch.float32)
    for i in (0, 1, 3, 4, 5):
        assert_close(rows(1 + i), torch.stack([full["a"][25 + i], full["b"][6 + i]][:2 if i < 4 else 1]), torch.float32)
    assert_close(rows(7), torch.stack([full["c"][19], full["d"][0], full["d"][8]]), torch.float32)


@pytest.mark.gpu
@pytest.mark.parametrize("name,dtype", [("tile", torch.bfloat16), ("odd", torch.float32), ("wide", torch.bfloat16)])
def test_branches_on_two_streams_change_nothing(tmp_path, cuda_device, name, dtype):
    """long prompts run a parallel layer's delta rule on a second stream while the attention runs on the first: the same kernels on the
    same numbers, so the logits are the same bit for bit, call after call, and decoding continues from the state such a prompt left"""
    from ipex_llm_b200.transformers.models import bugipel
    cfg, w, model = build(tmp_path, name, dtype, cuda_device)
    ids = torch.tensor([tokens_for(cfg, 130, s) for s in (1, 2, 3)], device=cuda_device)
    assert ids.numel() >= bugipel.OVERLAP_MIN_TOKENS
    with torch.no_grad():
        model.overlap_branches = False
        want = model(input_ids=ids, use_cache=True)
        want_next = model(input_ids=ids[:, :1], past_key_values=want.past_key_values, use_cache=True).logits
        model.overlap_branches = True
        for _ in range(4):
            got = model(input_ids=ids, use_cache=True)
            assert model._side_stream is not None and torch.equal(got.logits, want.logits)
        assert torch.equal(model(input_ids=ids[:, :1], past_key_values=got.past_key_values, use_cache=True).logits, want_next)
