"""The Rumuvik design in the framework against the plain statements of tests/rumuvik_oracle.py (float64).

CPU tests cover what needs no kernel: the configuration reader, the order of layer runs, the checkpoint's name map, the merged
projections, the latent expansion, the registry, the rotary frequencies, and properties of the oracle itself (rotated values see
distances only, the mLSTM's running maximum is a gauge).  GPU tests run the kernels (there is no CPU path): every mechanism alone on
odd sizes, then the model: whole prompts against token-by-token decoding and portions down to two tokens, unequal batches against
each request alone, rows leaving a batch, storage that grows and is used again, long decoding, far tokens, greedy generation through
``generate()`` and the trace runner's command line.
"""
import json
import math
import os
import subprocess

import pytest
import torch

import rumuvik_oracle as O

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
    # nothing coincides: fewer key than query heads, dim != vdim, head sizes that are no multiples of 8, a partly rotated head, a layer
    # without feed-forward inside the loop, feed-forwards of different widths, layers before and behind the loop
    "odd": dict(),
    # everything 1 or equal or absent: one head everywhere, the whole head rotated, no rescaled frequencies, scales of 1, no loop
    "plain": dict(width=32, vocab=40, order=("attention", "mlstm", "latent_attention"), ffs=(32, None, 32), att=dict(heads=1, kv_heads=1, dim=8, vdim=8, rot_dims=8,
                  scale=1.0, softcap=1.0), lat=dict(heads=1, dim=8, rot_dim=8, vdim=8, kv_rank=8, q_rank=8, scale=1.0, scaling=None),
                  mem=dict(heads=1, dim=8, vdim=8, gate_cap=1.0), loop=None, embed_scale=1.0),
    # head sizes that tile into 16s (the tensor-core attention of a 16-bit model); the loop covers every layer, twice
    "tile": dict(width=64, vocab=83, order=("latent_attention", "attention", "mlstm"), ffs=(40, None, 72), att=dict(heads=4, kv_heads=2, dim=48, vdim=32,
                 rot_dims=16, base=10000.0, scale=0.2, softcap=20.0), lat=dict(heads=4, dim=32, rot_dim=16, vdim=32, kv_rank=48, q_rank=64, base=10000.0),
                 mem=dict(heads=4, dim=32, vdim=64), loop=(0, 3, 2)),
    # heads of a served model on a narrow stream: four queries per key head of 128 and a latent of 128 (decoding takes the kernel that
    # splits the keys of shared heads over blocks), a wide recurrent head, a loop of one layer that ends the stack
    "wide": dict(width=72, vocab=300, order=("mlstm", "latent_attention", "attention"), ffs=(100, 24, 64), att=dict(heads=8, kv_heads=2, dim=128, vdim=128,
                 rot_dims=32, base=500000.0, scale=0.05, softcap=30.0), lat=dict(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=40, base=500000.0,
                 scale=0.1), mem=dict(heads=2, dim=136, vdim=24), loop=(2, 3, 4), embed_scale=7.0),
    # sizes that are multiples of nothing, a loop that runs once, a negative scale, latent layers in the loop
    "awkward": dict(width=52, vocab=37, order=("attention", "mlstm", "latent_attention"), ffs=(25, 11, None), att=dict(heads=3, kv_heads=3, dim=6, vdim=14,
                    rot_dims=2, base=7.0, scale=-0.3, softcap=2.0), lat=dict(heads=5, dim=3, rot_dim=2, vdim=7, kv_rank=9, q_rank=5, base=11.0,
                    scaling=dict(factor=2.0, original=40, fast=30.0, slow=20.0)), mem=dict(heads=5, dim=3, vdim=7, gate_cap=15.0), loop=(0, 1, 1), eps=1e-3),
}


def make(name, seed=0):
    cfg = O.random_config(**CONFIGS[name])
    return cfg, O.random_weights(cfg, seed + 1)


def w64(w):
    return {k: v.to(F64) for k, v in w.items()}


def tokens_for(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


# ================================================================== CPU: configuration, loader, order of layers, the oracle itself
def test_loader_maps_every_tensor_and_merges(tmp_path):
    cfg, w = make("odd")
    save_checkpoint(cfg, w, tmp_path)
    model = load_framework(tmp_path, torch.bfloat16)
    assert type(model).__name__ == "RumuvikForCausalLM" and model.config.model_type == "rumuvik"
    W = cfg["width"]
    layers = model.model.layers
    assert [l.kind for l in layers] == list(O.random_config()["layers"][i]["type"] for i in range(4)) and layers[2].mlp is None and not hasattr(layers[2], "norm2")
    assert torch.equal(model.lm_head.weight, w["head"]) and torch.equal(model.model.embed_tokens.weight, w["embed"]) and model.config.embedding_scale == 2.5
    a = layers[0].mixer                                                     # q 72 | k 24 | v 20
    assert a.in_proj.weight.shape == (116, W) and torch.equal(a.in_proj.weight[72:96], w["l0.mix.k"]) and torch.equal(a.in_proj.bias[96:], w["l0.mix.v.b"])
    assert (a.scale, a.softcap, a.rotary.dims, a.value_rotary.dims) == (0.5, 4.0, 8, 10) and a.value_rotary.freq[1] == pytest.approx(50.0 ** -0.2)
    assert layers[0].out_proj.weight.shape == (W, 60 + 24) and torch.equal(layers[0].out_proj.weight[:, 60:], w["l0.mlp.down"])
    assert torch.equal(layers[0].out_proj.weight[:, :60], w["l0.mix.o"]) and torch.equal(layers[0].mlp.gate_up.weight[24:], w["l0.mlp.up"])
    t = layers[1].mixer                                                     # query latent 22 | latent 18 | rotated part 6
    assert t.in_proj.weight.shape == (46, W) and torch.equal(t.in_proj.weight[22:], w["l1.mix.dkv"]) and t.in_proj.bias is None
    e = t.expand.weight                                                     # keys 4 x 16, values 4 x 14, rows of 18 + 6
    assert e.shape == (64 + 56, 24) and torch.equal(e[16:26, :18], w["l1.mix.uk"][10:20]) and torch.equal(e[64:, :18], w["l1.mix.uv"])
    assert torch.equal(e[26:32, 18:], torch.eye(6, dtype=e.dtype)) and not e[26:32, :18].any() and not e[:10, 18:].any() and not e[64:, 18:].any()
    m = layers[2].mixer                                                     # q, k: 30; v, gate: 42; two gates of 3
    assert m.in_proj.weight.shape == (144 + 6, W) and torch.equal(m.in_proj.weight[147:], w["l2.mix.f"]) and torch.equal(m.i_bias, w["l2.mix.i.b"])
    assert m.cap == 6.0 and torch.equal(layers[2].out_proj.weight, w["l2.mix.o"])
    # a missing tensor and tensors of the wrong shape are refused, by name
    for name, bad in (("l1.mix.dq.norm", None), ("l2.mix.i.b", torch.zeros(4, dtype=torch.bfloat16)), ("l1.mix.uk", torch.zeros(4, 18).bfloat16()),
                      ("l0.mix.q.b", None)):
        broken = dict(w)
        if bad is None:
            del broken[name]
        else:
            broken[name] = bad
        save_checkpoint(cfg, broken, tmp_path / "bad")
        with pytest.raises(RuntimeError, match="l1: the key|i_bias|" + name.replace(".", r"\.")):
            load_framework(tmp_path / "bad", torch.bfloat16)


def test_unsupported_configurations_are_refused(tmp_path):
    for change, text in ((lambda c: c["layers"][0]["mixer"].update(kv_heads=4), "kv_heads"), (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=14), "rotary"),
                         (lambda c: c["layers"][0]["mixer"].update(vdim=9), "even"), (lambda c: c["layers"][1].update(type="other"), "layer type"),
                         (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "feed-forward")):
        cfg, w = make("odd")
        change(cfg)
        save_checkpoint(cfg, w, tmp_path)
        with pytest.raises(RuntimeError, match=text):
            load_framework(tmp_path, torch.bfloat16)


def test_registry_picks_the_design(tmp_path):
    from ipex_llm_b200.transformers.model import native_architecture
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Rumuvik"}))
    assert native_architecture(tmp_path).endswith("models.rumuvik")


def test_order_of_layer_runs():
    from ipex_llm_b200.transformers.models.rumuvik import RumuvikConfig
    layers = [{"type": "mlstm"}] * 4
    assert RumuvikConfig(layers=layers).layer_runs() == [(0, False), (1, False), (2, False), (3, False)]
    got = RumuvikConfig(layers=layers, loop={"start": 1, "stop": 3, "times": 2}).layer_runs()
    assert got == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    assert RumuvikConfig(layers=layers, loop={"start": 3, "stop": 4, "times": 3}).layer_runs() == [(i, False) for i in range(4)] + [(3, True), (3, True)]
    for loop in (None, (1, 3, 2), (0, 4, 1), (3, 4, 3), (0, 4, 3)):
        cfg = {"layers": layers, "loop": loop and {"start": loop[0], "stop": loop[1], "times": loop[2]}}
        assert O.layer_runs(cfg) == RumuvikConfig(**cfg).layer_runs()
    with pytest.raises(RuntimeError):
        RumuvikConfig(layers=layers, loop={"start": 2, "stop": 5, "times": 2}).layer_runs()


def test_rescaled_frequencies_match_the_plain_statement():
    from ipex_llm_b200.transformers.models.mixers import Rotary
    for rot in ({"dims": 6, "base": 300.0, "scaling": dict(factor=3.0, original=64, fast=8.0, slow=1.0)}, {"dims": 16, "base": 1e4}, {"dims": 2, "base": 9.0},
                {"dims": 64, "base": 5e5, "scaling": dict(factor=40.0, original=4096, fast=32.0, slow=1.0)},
                {"dims": 8, "base": 11.0, "scaling": dict(factor=2.0, original=40, fast=30.0, slow=30.0)}):
        r = Rotary(rot)
        f, amp = O.rot_frequencies(rot)
        assert torch.allclose(torch.tensor(r.freq, dtype=F64), f, rtol=1e-12) and r.amp == pytest.approx(amp)


def test_oracle_rotated_values_see_distances_only():
    """shifting every position leaves the output alone (keys and values turn by their own position, the output turns back), and a
    sequence's first token returns its own value times its softmax weight"""
    g = torch.Generator().manual_seed(0)
    q, k, v = torch.randn(9, 4, 6, generator=g, dtype=F64), torch.randn(9, 2, 6, generator=g, dtype=F64), torch.randn(9, 2, 8, generator=g, dtype=F64)
    a = [O.turned_value_attention(q, k, v, torch.arange(9) + s, {"dims": 4, "base": 30.0}, 0.7, 3.0) for s in (0, 1000)]
    assert (a[0] - a[1]).abs().max() < 1e-10
    s = O.cap_scores((q[0] * k[0].repeat_interleave(2, 0)).sum(-1) * 0.7, 3.0)
    assert torch.allclose(a[0][0], torch.sigmoid(s)[:, None] * v[0].repeat_interleave(2, 0))
    plain = torch.einsum("hij,jhd->ihd", O.softmax_with_one(torch.zeros(4, 9, 9, dtype=F64)), v.repeat_interleave(2, 1))
    assert (a[0][8] - plain[8]).abs().max() > 0.1


def test_oracle_running_maximum_is_a_gauge():
    """the stabilised recurrence is the plain one (S without the maximum, denominator against 1) wherever that one does not overflow"""
    g = torch.Generator().manual_seed(1)
    T, H, D, Dv = 30, 2, 5, 4
    q, k, v = torch.randn(T, H, D, generator=g, dtype=F64), torch.randn(T, H, D, generator=g, dtype=F64), torch.randn(T, H, Dv, generator=g, dtype=F64)
    i, f = O.mlstm_gates(torch.randn(T, H, generator=g, dtype=F64) * 4, torch.randn(T, H, generator=g, dtype=F64) * 3 + 1, 5.0)
    got, _ = O.mlstm_scan(q, k, v, i, f)
    S, n = torch.zeros(H, D, Dv, dtype=F64), torch.zeros(H, D, dtype=F64)
    for t in range(T):
        S = f[t].exp()[:, None, None] * S + i[t].exp()[:, None, None] * k[t].unsqueeze(-1) * v[t].unsqueeze(-2)
        n = f[t].exp()[:, None] * n + i[t].exp()[:, None] * k[t]
        want = torch.einsum("hij,hi->hj", S, q[t]) / torch.clamp((n * q[t]).sum(-1).abs(), min=1.0)[:, None]
        assert (got[t] - want).abs().max() < 1e-4 * (1 + want.abs().max())
    # cut in two with the state handed over
    first, state = O.mlstm_scan(q[:11], k[:11], v[:11], i[:11], f[:11])
    second, _ = O.mlstm_scan(q[11:], k[11:], v[11:], i[11:], f[11:], state)
    assert torch.equal(torch.cat([first, second]), got)


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
                                          (3, 48, 31, (129,)), (20, 64, 64, (36, 20)), (2, 520, 8, (18, 2)), (5, 3, 200, (17, 16, 15)), (2, 16, 15, (40, 1, 1))])
def test_mlstm_with_carried_state(mixers, cuda_device, dtype, H, D, Dv, sizes):
    """the few-token and the pipelined kernel, matrix, normaliser and running maximum carried from call to call, a row whose first tokens
    are padding, columns out of the middle of a wider projection; input gates that jump by orders of magnitude (the maximum follows them
    up and decays), tokens whose read-out is below the floor of the denominator, and value counts around the kernels' column blocks"""
    g = torch.Generator().manual_seed(H * D + Dv)
    B, T, off, cap, tiny = 2, sum(sizes), 3, 9.0, 1e-6
    pads = [0, min(3, sizes[0] - 1)]
    offs = [off, off + H * D + 1, off + 2 * H * D + 1]
    off_i = offs[2] + H * Dv + 2
    off_f = off_i + H
    proj = torch.randn(B, T, off_f + H + 1, generator=g)
    proj[..., off_i:off_f] = proj[..., off_i:off_f] * 3 + (torch.rand(B, T, H, generator=g) < 0.1) * 12.0
    proj[..., off_f:off_f + H] = proj[..., off_f:off_f + H] * 3 + 2
    proj = proj.to(dtype).to(cuda_device)
    bias_i, bias_f = _rand((H,), g, dtype, cuda_device), _rand((H,), g, dtype, cuda_device)
    new = lambda *s: torch.zeros(*s, dtype=torch.float32, device=cuda_device)        # noqa: E731
    state, norm, top = new(B, H, D, Dv), new(B, H, D), new(B, H, Dv + 1)
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    outs, belows, at = [], [], 0
    for n in sizes:
        o, below = mixers.mlstm(proj[:, at:at + n].contiguous(), *offs, off_i, off_f, H, D, Dv, bias_i, bias_f, cap, tiny, state, norm, top, at,
                                pad if at == 0 else None)
        outs.append(o)
        belows.append(below)
        at += n
    o, below = _c64(torch.cat(outs, 1)), _c64(torch.cat(belows, 1))
    for b, p in enumerate(pads):
        c = _c64(proj[b, p:])
        n = T - p
        q, k, v = (c[:, a:a + H * d].reshape(n, H, d) for a, d in zip(offs, (D, D, Dv)))
        i, f = O.mlstm_gates(c[:, off_i:off_f] + _c64(bias_i), c[:, off_f:off_f + H] + _c64(bias_f), cap)
        want_o, want_below, (S, nrm, m) = O.mlstm_parts(q * D ** -0.5, k, v, i, f)
        assert (o[b, p:] - want_o).abs().max() / (want_o.abs().max() + 1) < 1e-5
        assert (below[b, p:] - want_below).abs().max() / (want_below.max() + 1) < 1e-5 and below.min() > 0
        assert (top[b].cpu().to(F64) - m[:, None]).abs().max() < 1e-4                # one number per head, the same for every column
        assert (_c64(state[b]) - S).abs().max() / (S.abs().max() + 1) < 2e-5 and (_c64(norm[b]) - nrm).abs().max() / (nrm.abs().max() + 1) < 2e-5
        assert o[b, :p].abs().sum() == 0 and (below[b, :p] == 1).all()


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_mlstm_floor_and_extreme_gates(mixers, cuda_device, dtype):
    """a key orthogonal to the query: the denominator is exp(-m) + tiny, whatever n holds; logits far outside the cap; a forget gate of
    almost nothing that wipes the state"""
    H, D, Dv, cap = 1, 4, 3, 5.0
    proj = torch.zeros(1, 3, 2 * D + Dv + 2)
    proj[0, :, 0], proj[0, :, D + 1] = 2.0, 3.0                              # q along the first axis, k along the second
    proj[0, :, 2 * D:2 * D + Dv] = torch.tensor([1.0, -2.0, 0.5])
    proj[0, :, -2] = torch.tensor([1000.0, -1000.0, 0.0])                    # input gates e^5, e^-5, 1
    proj[0, :, -1] = torch.tensor([0.0, 1000.0, -1000.0])
    proj[0, 2, 1] = 1.0                                                      # the last query sees the stored key
    dev = proj.to(dtype).to(cuda_device)
    zero = torch.zeros(H, dtype=dtype, device=cuda_device)
    st = [torch.zeros(s, dtype=torch.float32, device=cuda_device) for s in ((1, H, D, Dv), (1, H, D), (1, H, Dv + 1))]
    o, below = mixers.mlstm(dev, 0, D, 2 * D, 2 * D + Dv, 2 * D + Dv + 1, H, D, Dv, zero, zero, cap, 1e-6, *st, 0, None)
    i, f = O.mlstm_gates(_c64(dev[0, :, -2:-1]), _c64(dev[0, :, -1:]), cap)
    m1 = max(f[0].item(), 5.0)
    assert below[0, 0, 0].item() == pytest.approx(math.exp(-m1) + 1e-6, rel=1e-5)
    m2 = max(f[1].item() + m1, i[1].item())
    assert below[0, 1, 0].item() == pytest.approx(math.exp(-m2) + 1e-6, rel=1e-5)
    want, _ = O.mlstm_scan(_c64(dev[0, :, :D]).view(3, H, D) * D ** -0.5, _c64(dev[0, :, D:2 * D]).view(3, H, D), _c64(dev[0, :, 2 * D:2 * D + Dv]).view(3, H, Dv), i, f)
    assert (_c64(o / below.unsqueeze(-1))[0] - want).abs().max() < 1e-5 and want[2].abs().max() > 0.1


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("n,H,Dv", [(7, 3, 14), (5, 4, 300), (1500, 2, 520), (2, 3, 1030), (4, 2, 2052), (1300, 8, 256)])
def test_head_norm_of_a_read_out_over_its_denominator(mixers, cuda_device, dtype, n, H, Dv):
    """denominators from 1e-5 to 1e3 and an eps that matters: dividing behind the norm, or not at all, would show"""
    g = torch.Generator().manual_seed(n)
    eps = 1e-2
    o = torch.randn(n, H, Dv, generator=g)
    below = 10.0 ** (torch.rand(n, H, generator=g) * 8 - 5)
    o = (o * below.unsqueeze(-1) * 10.0 ** (torch.rand(n, H, 1, generator=g) * 3 - 2)).to(cuda_device)
    gate, w = _rand((n, H * Dv + 4), g, dtype, cuda_device), _rand((H * Dv,), g, dtype, cuda_device) + 1.0
    for off in (4, 3):
        out = torch.full((n, H * Dv + 8), 7.0, dtype=dtype, device=cuda_device)
        mixers.gated_rms_norm(o, gate, off, w, eps, out, 4, 1.0, sigmoid=True, below=below.to(cuda_device))
        want = O.unit_rms(_c64(o) / below.to(F64).unsqueeze(-1), eps).reshape(n, -1) * _c64(w) * torch.sigmoid(_c64(gate[:, off:off + H * Dv]))
        assert (out[:, :4] == 7).all() and (out[:, 4 + H * Dv:] == 7).all()
        assert ((_c64(out[:, 4:4 + H * Dv]) - want).abs() / (1 + want.abs())).max() < (1e-5 if dtype == torch.float32 else 0.02)
    without = O.unit_rms(_c64(o), eps).reshape(n, -1) * _c64(w) * torch.sigmoid(_c64(gate[:, off:off + H * Dv]))
    assert (without - want).abs().max() > 0.1


@pytest.mark.gpu
@pytest.mark.parametrize("amp,dims,base", [(1.0, 8, 50.0), (1.3, 66, 5e5), (1.0, 2, 3.0)])
def test_table_of_angles(mixers, cuda_device, amp, dims, base):
    """near and far positions, padding, the slot number read from the device"""
    f = O.plain_frequencies(dims, base)
    pad = torch.tensor([0, 3], dtype=torch.int32, device=cuda_device)
    B, S = 2, 7
    for held, shift, dyn in ((0, 0, None), (5, 100000, None), (1, 0, 40)):
        word = None if dyn is None else torch.tensor([dyn], dtype=torch.int32, device=cuda_device)
        t = _c64(mixers.rotary_table(f.to(cuda_device), amp, B, S, held, shift, pad, dyn=word)).view(B, S, dims // 2, 2)
        for b in range(B):
            pos = torch.arange(S) + (held if dyn is None else dyn) + shift - int(pad[b])
            want = torch.stack([torch.cos(pos[:, None] * f), torch.sin(pos[:, None] * f)], -1) * amp
            want[pos < 0] = 0
            assert (t[b] - want).abs().max() < 3e-7


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("held,shift", [(0, 0), (6, 4000)])
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("H,G,D,Dv,dims", [(6, 2, 12, 10, 8), (3, 3, 10, 66, 10), (4, 1, 64, 64, 0), (2, 2, 130, 2, 128)])
def test_rotated_queries_keys_and_values_enter_the_cache(mixers, cuda_device, dtype, held, shift, interleaved, H, G, D, Dv, dims):
    """both pairings; keys and values out of another buffer than the queries; far positions keep their angle, padding slots hold zeros,
    neighbours in the cache stay untouched"""
    g = torch.Generator().manual_seed(D)
    B, S, cap, base, amp = 2, 5, 16, 50.0, 1.2
    pads = [0, 2]
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    tol = 2e-5 if dtype == torch.float32 else 0.04
    f, vf = O.plain_frequencies(dims, base) if dims else torch.zeros(0, dtype=F64), O.plain_frequencies(Dv, base)
    table = mixers.rotary_table(f.to(cuda_device), amp, B, S, held, shift, pad) if dims else None
    v_table = mixers.rotary_table(vf.to(cuda_device), 1.0, B, S, held, shift, pad)
    qp, kvp = _rand((B, S, H * D + 3), g, dtype, cuda_device), _rand((B, S, 1 + G * D + 2 + G * Dv), g, dtype, cuda_device)
    ks, vs = torch.full((B, G, cap, D), 9.0, dtype=dtype, device=cuda_device), torch.full((B, G, cap, Dv), 9.0, dtype=dtype, device=cuda_device)
    q = mixers.rope_qk_prepare(qp, 0, 1, 1 + G * D + 2, H, G, D, D, Dv, 0, 0, dims, None, 1.0, ks, (G * cap * D, D, cap * D), vs, (G * cap * Dv, Dv, cap * Dv),
                               held, shift, pad, table=table, v_table=v_table, interleaved=interleaved, kv_proj=kvp)
    for b in range(B):
        first = max(pads[b] - held - shift, 0)
        pos = torch.arange(S) + held + shift - pads[b]
        kv = _c64(kvp[b])
        for got, raw, freq, a in ((q.view(B, S, H, D)[b], _c64(qp[b, :, :H * D]).view(S, H, D), f, amp),
                                  (ks[b, :, held:held + S].transpose(0, 1), kv[:, 1:1 + G * D].reshape(S, G, D), f, amp),
                                  (vs[b, :, held:held + S].transpose(0, 1), kv[:, 3 + G * D:].reshape(S, G, Dv), vf, 1.0)):
            want = O.turn(raw, pos, freq, a, interleaved)
            assert (_c64(got)[first:] - want[first:]).abs().max() < tol
            assert _c64(got)[:first].abs().sum() == 0
        for t in (ks, vs):
            assert (t[b, :, :held] == 9).all() and (t[b, :, held + S:] == 9).all()


ATTENTION = [(torch.float32, 5, 0, 6, 2, 5, 6, False), (torch.float32, 1, 300, 4, 1, 24, 40, False), (torch.float32, 2, 9, 2, 1, 8, 1034, False),
             (torch.bfloat16, 1, 517, 3, 1, 64, 64, False), (torch.bfloat16, 40, 30, 4, 2, 32, 16, True), (torch.float16, 150, 0, 3, 1, 64, 48, True),
             (torch.bfloat16, 70, 3, 2, 1, 96, 96, True), (torch.bfloat16, 33, 0, 2, 1, 128, 128, True), (torch.bfloat16, 66, 0, 2, 2, 16, 112, True),
             (torch.bfloat16, 20, 5, 2, 1, 144, 240, True), (torch.bfloat16, 1, 700, 8, 2, 128, 128, True), (torch.bfloat16, 3, 130, 4, 1, 32, 256, True)]


@pytest.mark.gpu
@pytest.mark.parametrize("interleaved", [False, True])
@pytest.mark.parametrize("dtype,S,held,H,G,D,Dv,tc", ATTENTION)
def test_outputs_are_turned_back_in_every_attention_kernel(mixers, cuda_device, dtype, S, held, H, G, D, Dv, tc, interleaved):
    """the general kernel, the prompt kernel on the tensor cores and the split-key kernel, written into the middle of a wider buffer,
    with capped scores and the one in the denominator; keys and values as they lie in the cache (values rotated)"""
    g = torch.Generator().manual_seed(S + held)
    B, L, scale, cap = 2, held + S, 1.5 / D ** 0.5, 3.0
    k, raw_v = _rand((B, L, G, D), g, dtype, cuda_device), torch.randn(B, L, G, Dv, generator=g)
    q = _rand((B * S, H * D), g, dtype, cuda_device)
    pads = [0, min(L - 1, 3)]
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    f = O.plain_frequencies(Dv, 100.0)
    v = torch.stack([O.turn(raw_v[b].to(F64), torch.arange(L) - pads[b], f, 1.0, interleaved) for b in range(B)]).to(dtype).to(cuda_device)
    back = mixers.rotary_table(f.to(cuda_device), 1.0, B, S, held, 0, pad)
    out = torch.full((B * S, H * Dv + 24), 7.0, dtype=dtype, device=cuda_device)
    mixers.softmax_attention(q, k, v, B, S, H, held, 0, pad, 0, scale, out=out, out_col=8, tensor_cores=tc, softcap=cap,
                             sink=torch.zeros(H, dtype=dtype, device=cuda_device), back=back, back_interleaved=interleaved)
    assert (out[:, :8] == 7).all() and (out[:, 8 + H * Dv:] == 7).all()
    got = _c64(out[:, 8:8 + H * Dv]).view(B, S, H, Dv)
    for b in range(B):
        for t in range(S):
            c, p = held + t, pads[b]
            if c < p:
                assert got[b, t].abs().sum() == 0
                continue
            for h in range(H):
                s = O.cap_scores(_c64(k[b, p:c + 1, h // (H // G)]) @ _c64(q.view(B, S, H, D)[b, t, h]) * scale, cap)
                sums = O.softmax_with_one(s) @ _c64(v[b, p:c + 1, h // (H // G)])
                want = O.turn(sums.view(1, 1, Dv), torch.tensor([c - p]), f, 1.0, interleaved, back=True)[0, 0]
                assert (got[b, t, h] - want).abs().max() < (2e-5 if dtype == torch.float32 else 0.03)
    assert held + S < 4 or (sums - want).abs().max() > 0.01


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,S,tc", [(torch.float32, 1, False), (torch.float32, 40, False), (torch.bfloat16, 1, False), (torch.bfloat16, 40, True),
                                        (torch.bfloat16, 1, True), (torch.bfloat16, 9, True)])
def test_one_outstanding_key_anywhere(mixers, cuda_device, dtype, S, tc):
    """a key whose capped score dwarfs all others (and the sink): its value, turned by the distance, is the output wherever it sits -- the
    first token, the borders of the kernels' key tiles, far back, the query itself -- and it must not show from the future or from in
    front of the row's first token"""
    g = torch.Generator().manual_seed(11)
    H, D, Dv, L = 4, 16, 128, 1300
    held = L - S
    base_k, base_v = torch.randn(1, L + 8, 1, D, generator=g) * 0.1, torch.randn(1, L + 8, 1, Dv, generator=g)
    spike = torch.zeros(D)
    spike[3] = 40.0
    q = (torch.randn(S, H * D, generator=g) * 0.1 + spike.repeat(H)[None]).to(dtype).to(cuda_device)
    f = O.plain_frequencies(Dv, 1000.0)
    none = torch.zeros(1, dtype=torch.int32, device=cuda_device)
    v_dev = O.turn(base_v[0].to(F64), torch.arange(L + 8), f)[None].to(dtype).to(cuda_device)
    back = mixers.rotary_table(f.to(cuda_device), 1.0, 1, S, held, 0, none)
    zero = torch.zeros(H, dtype=dtype, device=cuda_device)

    def shows(at, query=S - 1, first=0):
        k = base_k.clone()
        k[0, at, 0] = spike
        out = mixers.softmax_attention(q, k.to(dtype).to(cuda_device), v_dev, 1, S, H, held, 0, torch.tensor([first], dtype=torch.int32, device=cuda_device),
                                       0, 1.0, tensor_cores=tc, sink=zero, softcap=25.0, back=back)
        want = O.turn(base_v[0, at].to(F64)[None], torch.tensor([held + query - at]), f, back=True)[0, 0]
        d = (out.float().cpu().view(S, H, Dv)[query] - want).abs().max()
        assert d < 0.04 or d > 0.3, d
        return bool(d < 0.04)

    for at in (0, 1, 31, 32, 63, 64, 255, 256, 257, 511, 512, 1023, 1024, L - 2, L - 1):
        assert shows(at), at
    assert not shows(L) and not shows(4, first=5) and shows(5, first=5)
    if S > 21:
        assert shows(held + 20, query=20) and not shows(held + 21, query=20) and shows(held + 21, query=21)


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,D,Dr,Dv,R,sizes", [(3, 10, 6, 14, 18, (20, 1, 16, 17, 2)), (4, 32, 16, 32, 48, (33, 1, 1)), (8, 64, 32, 64, 128, (130, 1, 9)), (1, 1, 2, 1, 1, (4, 30))])
def test_latent_attention_few_and_many_tokens(mixers, cuda_device, dtype, H, D, Dr, Dv, R, sizes):
    """the query latent's norm (columns out of a wider projection, an eps that matters), the cache rows [normed latent | rotated shared
    part] with neighbouring pairs, then attention on the cache itself (up to 16 new tokens) and on the expanded keys and values"""
    from ipex_llm_b200.transformers.models.mixers import ABSORB_MAX_TOKENS, latent_cache_attention, latent_expansion
    assert ABSORB_MAX_TOKENS == 16
    g = torch.Generator().manual_seed(R)
    B, T, Q, eps, scale, base, amp = 2, sum(sizes), 12, 0.05, 0.8 / (D + Dr) ** 0.5, 40.0, 1.15
    pads = [0, min(2, sizes[0] - 1)]
    pad = torch.tensor(pads, dtype=torch.int32, device=cuda_device)
    proj = _rand((B, T, Q + R + Dr), g, dtype, cuda_device)
    wq, wc, uq = _rand((Q,), g, dtype, cuda_device, 0.3) + 1, _rand((R,), g, dtype, cuda_device, 0.3) + 1, _rand((H * (D + Dr), Q), g, dtype, cuda_device, 0.5)
    uk, uv = _rand((H * D, R), g, dtype, "cpu", 1 / R ** 0.5), _rand((H * Dv, R), g, dtype, "cpu", 1 / R ** 0.5)
    expand = latent_expansion(uk, uv, H, D, Dr, Dv, R).to(cuda_device)
    f = O.plain_frequencies(Dr, base)
    store = torch.full((B, T + 3, R + Dr), 9.0, dtype=dtype, device=cuda_device)
    got, at = [], 0
    for n in sizes:
        part = proj[:, at:at + n].contiguous()
        cq = mixers.rms_norm_columns(part, 0, Q, wq, eps, at, 0, pad)
        q = torch.nn.functional.linear(cq, uq)
        q = mixers.rope_qk_prepare(q.view(B, n, -1), 0, Q, 0, H, 1, D + Dr, R + Dr, 0, D, R, Dr, None, 1.0, store, (store.stride(0), R + Dr, 0), None, None, at, 0,
                                   pad, eps=eps, k_norm_w=wc, k_norm_cols=R, table=mixers.rotary_table(f.to(cuda_device), amp, B, n, at, 0, pad), interleaved=True,
                                   kv_proj=part)
        out = torch.full((B * n, H * Dv + 5), 7.0, dtype=dtype, device=cuda_device)
        latent_cache_attention(q, expand, store, B, n, H, D + Dr, Dv, R, at, 0, pad, scale, out)
        assert (out[:, H * Dv:] == 7).all()
        got.append(_c64(out[:, :H * Dv]).view(B, n, H, Dv))
        at += n
    got = torch.cat(got, 1)
    assert (store[:, T:] == 9).all()
    for b, p in enumerate(pads):
        c = _c64(proj[b, p:])
        n = T - p
        pos = torch.arange(n)
        q = ((O.unit_rms(c[:, :Q], eps) * _c64(wq)) @ _c64(uq).T).view(n, H, D + Dr)
        lat = O.unit_rms(c[:, Q:Q + R], eps) * _c64(wc)
        shared, qr = O.turn(c[:, None, Q + R:], pos, f, amp, True)[:, 0], O.turn(q[..., D:], pos, f, amp, True)
        assert (_c64(store[b, p:T]) - torch.cat([lat, shared], -1)).abs().max() < (1e-5 if dtype == torch.float32 else 0.03)
        s = torch.einsum("ihd,jhd->hij", q[..., :D], (lat @ uk.to(F64).T).view(n, H, D)) + torch.einsum("ihd,jd->hij", qr, shared)
        pr = torch.softmax((s * scale).masked_fill(~O.causal(n)[None], float("-inf")), -1)
        want = torch.einsum("hij,jhd->ihd", pr, (lat @ uv.to(F64).T).view(n, H, Dv))
        assert (got[b, p:] - want).abs().max() < (5e-5 if dtype == torch.float32 else 0.06)
        assert got[b, :p].abs().sum() == 0


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
def test_tanh_gelu_product(mixers, cuda_device, dtype):
    """columns that come in fours and that do not, into a column range of a wider buffer, arguments from far below to far above zero"""
    g = torch.Generator().manual_seed(2)
    for n, cols, extra in ((5, 13, 0), (3, 64, 4), (70000, 8, 0), (9, 1000, 3), (2, 4, 8)):
        gu = _rand((n, 2 * cols + extra), g, dtype, cuda_device, 3.0)
        gu[0, :4] = torch.tensor([-300.0, 300.0, 0.0, -6.0])
        buf = torch.full((n, 8 + cols + extra), 7.0, dtype=dtype, device=cuda_device)
        mixers.gelu_tanh_mul(gu, cols, out=buf[:, 8:8 + cols])
        want = O.gelu_tanh(_c64(gu[:, :cols])) * _c64(gu[:, cols:2 * cols])
        assert (buf[:, :8] == 7).all() and (buf[:, 8 + cols:] == 7).all()
        tol = {torch.float32: 2e-6, torch.bfloat16: 6e-3, torch.float16: 1e-3}[dtype]
        assert ((_c64(buf[:, 8:8 + cols]) - want).abs() / (1 + want.abs())).max() < tol
        assert torch.equal(mixers.gelu_tanh_mul(gu, cols), buf[:, 8:8 + cols])


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,n", [(45, 5), (1100, 3), (352, 1500), (8200, 2), (2000, 70), (1, 4)])
def test_residual_update_with_norms_stored_around_zero(mixers, cuda_device, dtype, width, n):
    """x += 32-bit product + embedding output, then two norms whose weights are 1 + w with w too small for a 16-bit 1 + w to hold; one
    number as the weight; and the lone norm in front of the head"""
    g = torch.Generator().manual_seed(width)
    eps = 1e-3
    x0 = torch.randn(n, width, generator=g) * 2 + 0.5
    y, again = _rand((n, width), g, torch.float32, cuda_device), _rand((n, width), g, torch.float32, cuda_device)
    w1, w2 = _rand((width,), g, dtype, cuda_device, 0.001), _rand((width,), g, dtype, cuda_device, 0.4)
    x = x0.clone().to(cuda_device)
    h1, h2 = mixers.sum_residual_norms(x, [y, again], dtype, eps, gain1=w1, gain2=w2, gain_add=1.0)
    new = x0.to(F64) + _c64(y) + _c64(again)
    assert (_c64(x) - new).abs().max() < 1e-5
    for got, w in ((h1, w1), (h2, w2), (mixers.rms_norm_rows(x, None, w1, eps, dtype, vec_add=1.0), w1)):
        want = O.zero_centred_norm(new, _c64(w), eps)
        d = (_c64(got) - want).abs() / (0.05 + want.abs())
        assert d.max() < (5e-5 if dtype == torch.float32 else 4.5e-3), d.max()          # bf16: little more than the result's own rounding
    one = _rand((1,), g, dtype, cuda_device, 0.3)
    x = x0.clone().to(cuda_device)
    h, _ = mixers.sum_residual_norms(x, [], dtype, eps, gain1=one[0], gain_add=1.0)
    want = O.zero_centred_norm(x0.to(F64), _c64(one), eps)
    assert (_c64(h) - want).abs().max() < (3e-5 if dtype == torch.float32 else 0.04)


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
    cfg = O.random_config(eps=0.05)                     # an mLSTM's head norm hides its denominator but for the norm's eps
    w = O.random_weights(cfg, 1)
    save_checkpoint(cfg, w, tmp_path)
    w, model = w64(w), load_framework(tmp_path, torch.float32, cuda_device)
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

    turn = O.turn

    def scan_without(what):
        def scan(q, k, v, i, f, state=None):
            T, H, D = q.shape
            S, n, m, out = torch.zeros(H, D, v.shape[-1], dtype=q.dtype), torch.zeros(H, D, dtype=q.dtype), torch.zeros(H, dtype=q.dtype), []
            for t in range(T):
                new = torch.maximum(f[t] + m, i[t])
                keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
                m = new
                S, n = keep[:, None, None] * S + take[:, None, None] * k[t].unsqueeze(-1) * v[t].unsqueeze(-2), keep[:, None] * n + take[:, None] * k[t]
                low = torch.ones_like(m) if what == "floor of one" else torch.exp(-m)
                d = (n * q[t]).sum(-1)
                d = (d if what == "sign" else d.abs())
                out.append(torch.einsum("hij,hi->hj", S, q[t]) / (torch.maximum(d, low) if what != "no floor" else d + 1e-3)[:, None])
            return torch.stack(out), None
        return scan

    assert moved() < 3e-5
    assert moved(softmax_with_one=lambda s: torch.softmax(s, -1)) > 1e-3                                 # the sink left out
    assert moved(cap_scores=lambda s, cap: s) > 1e-3
    assert moved(turn=lambda x, p, f, amp=1.0, interleaved=False, back=False: x if back else turn(x, p, f, amp, interleaved)) > 1e-3      # not turned back
    assert moved(turn=lambda x, p, f, amp=1.0, interleaved=False, back=False: turn(x, p, f, amp, False, back)) > 1e-3   # the other pairing
    assert moved(turn=lambda x, p, f, amp=1.0, interleaved=False, back=False: turn(x, p, f, 1.0, interleaved, back)) > 1e-3   # no amplitude
    assert moved(plain_frequencies=lambda dims, base, dtype=F64: torch.zeros(dims // 2, dtype=dtype)) > 1e-3
    assert moved(enter_pass=lambda x, x0: x) > 1e-3
    assert moved(zero_centred_norm=lambda x, wt, eps: O.unit_rms(x, eps) * wt) > 1e-3
    assert moved(gelu_tanh=lambda z: 0.5 * z * (1 + torch.erf(z / 2 ** 0.5))) > 1e-4
    assert moved(mlstm_gates=lambda i, f, cap: (i, torch.nn.functional.logsigmoid(f))) > 1e-4             # no cap
    for what in ("floor of one", "no floor", "sign"):
        assert moved(mlstm_scan=scan_without(what)) > 1e-3, what
    assert moved(change_cfg=lambda c: c["layers"][1]["mixer"]["rot"].pop("scaling")) > 1e-3
    assert moved(change_cfg=lambda c: c["loop"].update(times=2)) > 1e-3
    assert moved(change_cfg=lambda c: c["embedding"].update(scale=1.0)) > 1e-3
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l0.mix.v.b", "l2.mix.i.b", "l2.mix.f.b"):
        assert moved(change_w=lambda x: x.update({name: torch.zeros_like(x[name])})) > 1e-3, name
    for name in ("l1.mix.dq.norm", "l1.mix.dkv.norm", "l2.mix.norm"):
        assert moved(change_w=lambda x: x.update({name: torch.ones_like(x[name])})) > 1e-3, name


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
    are carried 300 times; the same request in portions around the store's block size"""
    cfg, w, model = build(tmp_path, "tile", torch.float32, cuda_device)
    tokens = tokens_for(cfg, 305, 9)
    want = O.forward(cfg, w, tokens)
    assert_close(run_portions(model, tokens, [5, 1], cuda_device), want, torch.float32)
    for sizes in ([255, 2, 48], [256, 1, 1, 47], [257, 48], [15, 16, 17, 2]):
        assert_close(run_portions(model, tokens, sizes, cuda_device), want, torch.float32)


@pytest.mark.gpu
@pytest.mark.parametrize("kind", ["attention", "latent_attention", "mlstm"])
def test_a_far_token_reaches_the_last_logits(tmp_path, cuda_device, kind):
    """changing one early token of a long prompt changes the last position's logits exactly as the plain statement says, in a prompt and
    when the tail is decoded token by token, through each mixer alone: the attention sees everything, the matrix memory hardly forgets"""
    cfg = O.random_config(order=(kind,), ffs=(None,), loop=(0, 1, 2) if kind != "mlstm" else None,
                          att=dict(heads=4, kv_heads=2, dim=8, vdim=8, rot_dims=2, base=1e9, scale=1.5, softcap=8.0),
                          lat=dict(base=1e9, scale=1.0, scaling=None))
    w = O.random_weights(cfg, 5)
    for k in w:
        if k.endswith("mix.f.b"):
            w[k] = w[k] + 30.0                                               # the cap holds the logit: a forget gate near sigmoid(6)
    folder = tmp_path / kind
    save_checkpoint(cfg, w, folder)
    w, model = w64(w), load_framework(folder, torch.float32, cuda_device)
    tokens = tokens_for(cfg, 260, 13)
    for at in (0, 1, 37):
        other = list(tokens)
        other[at] = (other[at] + 1) % cfg["vocab"]
        want_a, want_b = O.forward(cfg, w, tokens)[-1:], O.forward(cfg, w, other)[-1:]
        moved = position_errors(want_a, want_b).max()
        assert moved > 5e-5                                                 # the early token matters
        for sizes in ([260], [200, 1], [2, 258]):
            assert position_errors(run_portions(model, other, sizes, cuda_device)[-1:], want_b).max() < min(2e-5, 0.1 * moved)


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
    """a bf16 model whose attention and latent attention decode through the kernel that splits the keys of shared heads over blocks: the
    replayed step reads lengths and positions from the device, runs its feed-forwards on a second stream and must produce the tokens of
    the loop that passes everything from the host; every pass's states are updated in place by both"""
    cfg, w, model = build(tmp_path, "wide", torch.bfloat16, cuda_device)
    from ipex_llm_b200.ggml.model import mixers_cpp
    for heads, groups, dim in ((8, 2, 128), (4, 1, 160)):
        assert mixers_cpp.lib().mixers_softmax_attention_workspace(mixers_cpp.dtype_code(torch.bfloat16), 2, 1, heads, groups, dim, 128) > 0
    prompts = torch.tensor([tokens_for(cfg, 150, 1), [0] * 30 + tokens_for(cfg, 120, 2)], device=cuda_device)
    mask = torch.tensor([[1] * 150, [0] * 30 + [1] * 120], device=cuda_device)
    replayed = model.generate(prompts, attention_mask=mask, max_new_tokens=80, do_sample=False)
    assert model.__dict__.get("_b200_state_graph_failed") is None and model.__dict__.get("_b200_state_graphs") and model._side_stream is not None
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
    """the projections are ordinary linears to the converter: a sym_int4 model answers close to the 16-bit one; saved and loaded again it
    gives the same logits"""
    from ipex_llm_b200.transformers import AutoModelForCausalLM
    from ipex_llm_b200.transformers.low_bit_linear import LowBitLinear
    cfg = O.random_config(width=128, vocab=90, order=("attention", "latent_attention", "mlstm"), ffs=(192, 64, 128), mem=dict(heads=2, dim=32, vdim=64),
                          att=dict(heads=4, kv_heads=2, dim=32, vdim=32, rot_dims=32), lat=dict(heads=2, dim=32, rot_dim=32, vdim=64, kv_rank=64, q_rank=64),
                          loop=(0, 2, 2))
    w = O.random_weights(cfg, 3)
    save_checkpoint(cfg, w, tmp_path / "m")
    ref = load_framework(tmp_path / "m", torch.bfloat16, cuda_device)
    low = load_framework(tmp_path / "m", torch.bfloat16, None, load_in_low_bit="sym_int4").to(cuda_device)
    l = low.model.layers
    assert all(isinstance(m, LowBitLinear) for m in (l[0].mixer.in_proj, l[0].out_proj, l[1].mixer.uq, l[1].mlp.gate_up, l[2].mixer.in_proj, low.lm_head))
    assert low.model.embed_tokens.weight.dtype == l[1].mixer.expand.weight.dtype == torch.bfloat16
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
def test_feed_forward_on_a_second_stream_changes_nothing(tmp_path, cuda_device, name, dtype):
    """long prompts run a layer's feed-forward on a second stream while the mixer runs on the first: the same kernels on the same
    numbers, so the logits are the same bit for bit, call after call, and decoding continues from the state such a prompt left"""
    from ipex_llm_b200.transformers.models import rumuvik
    cfg, w, model = build(tmp_path, name, dtype, cuda_device)
    ids = torch.tensor([tokens_for(cfg, 130, s) for s in (1, 2, 3)], device=cuda_device)
    assert ids.numel() >= rumuvik.OVERLAP_MIN_TOKENS
    with torch.no_grad():
        model.overlap_feed_forward = False
        want = model(input_ids=ids, use_cache=True)
        want_next = model(input_ids=ids[:, :1], past_key_values=want.past_key_values, use_cache=True).logits
        model.overlap_feed_forward = True
        for _ in range(4):
            got = model(input_ids=ids, use_cache=True)
            assert model._side_stream is not None and torch.equal(got.logits, want.logits)
        assert torch.equal(model(input_ids=ids[:, :1], past_key_values=got.past_key_values, use_cache=True).logits, want_next)
