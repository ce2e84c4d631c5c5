"""Ketolix on the hybrid engine against the plain float64 statement of the design (`ketolix_oracle.py`).

Small configurations with random weights; every test builds its own.  The float32 engine is held to a tight bound, the
bfloat16 engine to the error that rounding its operands causes.
"""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

pytestmark = pytest.mark.gpu

from jax_llama_b200.config import KetolixConfig                                   # noqa: E402
from jax_llama_b200.generation import LLaMA                                       # noqa: E402
from jax_llama_b200.models.hybrid_engine import HybridEngine, random_tensors      # noqa: E402
from jax_llama_b200.models.ketolix import KetolixForCausalLM                      # noqa: E402
from jax_llama_b200.ops import seq_kernels as SK                                  # noqa: E402
from jax_llama_b200.tokenizers import IdTokenizer                                 # noqa: E402

from tests import ketolix_oracle as O                                             # noqa: E402

TOL = {torch.float32: 3e-4, torch.bfloat16: 8e-2}
DTYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def tol(dtype, cfg):
    """Rounding the operands of every layer to bfloat16 adds up along the stack: the bound grows with the layers beyond four."""
    return TOL[dtype] * (max(1.0, len(cfg.layers) / 4.0) if dtype == torch.bfloat16 else 1.0)


SCALING = {"factor": 4.0, "low": 1.0, "high": 3.0, "original": 64}


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def rotation(rot, base, scaling):
    r = {"dims": rot, "base": base}
    if scaling:
        r["scaling"] = dict(scaling)
    return r


def att(heads=4, kv_heads=2, dim=16, vdim=12, window=20, scale=0.3, cap=5.0, rot=8, base=100.0, scaling=SCALING, mix=True, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": mix}
    if cap:
        m["softcap"] = cap
    if window:
        m["mask"] = {"size": window}
    if rot:
        m["rot"] = rotation(rot, base, scaling)
    return {"type": "attention", "mixer": m, "mlp": mlp}


def par(heads=4, kv_heads=2, dim=12, window=15, scale=0.25, conv=3, rot=4, base=50.0, scaling=None, right=(3, 10, 14), ls=0.7, rs=0.4,
        decay=None, mlp=None):
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale, "conv": conv}
    if window:
        left["mask"] = {"size": window}
    if rot:
        left["rot"] = rotation(rot, base, scaling)
    H, D, Dv = right
    decay = decay or [1.0 - 0.6 / 3.0 ** h for h in range(H)]
    return {"type": "parallel", "mixer": {"left": left, "left_scale": ls, "right_scale": rs,
                                          "right": {"heads": H, "dim": D, "vdim": Dv, "decay": decay}}, "mlp": mlp}


def mem(heads=3, dim=20, vdim=18, cap=9.0, mlp=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp}


def config(layers, vocab=96, width=72, eps=1e-5):
    return KetolixConfig.from_dict({"architecture": "Ketolix", "vocab": vocab, "width": width, "norm": {"eps": eps},
                                    "layers": json.loads(json.dumps(layers))})


MIXED = [mem(mlp=dense()), att(mlp=dense()), par(mlp=dense(24)), att(heads=2, dim=10, window=33, rot=10, base=7.0, scaling=None),
         att(heads=6, kv_heads=3, vdim=8, window=0, cap=0.0, mix=False, mlp=dense(56))]


def build(cfg, dtype, seed=0, graph=True, tweak=None):
    tensors = random_tensors(cfg, "cuda", seed)
    g = torch.Generator(device="cuda").manual_seed(seed + 1000)

    def rnd(name, mean, std):
        tensors[name] = (mean + std * torch.randn(tensors[name].shape, device="cuda", generator=g)).to(torch.bfloat16)

    for name in list(tensors):
        if "norm" in name:
            rnd(name, 1.0, 0.3)
        if name.endswith("mix.sink"):                                    # sinks that take from nothing to most of the weight
            rnd(name, 0.0, 2.0)
        if name.endswith("vmix"):
            rnd(name, 0.45, 0.1)
        if name.endswith(("q.b", "k.b", "o.b")):
            rnd(name, 0.0, 0.5)
        if name.endswith("mix.i.b"):
            rnd(name, 0.0, 2.0)
        if ".conv" in name:
            rnd(name, 0.0, 0.6)
    if tweak is not None:
        tweak(tensors)
    eng = HybridEngine(cfg, tensors, dtype=dtype, device="cuda", use_cuda_graph=graph)
    return eng, {k: v.cpu() for k, v in tensors.items()}


def err(got, want):
    """Centred RMS difference over the vocabulary relative to the RMS of the wanted logits, worst row."""
    got, want = got.double().cpu(), want.double().cpu()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    return float((d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)).max())


def tokens(n, vocab, seed):
    return torch.randint(1, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def oracle_logits(cfg, cpu_tensors, toks, streams=None):
    return O.forward(toks, cpu_tensors, cfg.to_dict(), streams)


def feed(vals):
    return torch.tensor(vals, dtype=torch.int32).pin_memory()


def i32(vals):
    return torch.tensor(vals, dtype=torch.int32, device="cuda")


def decode_rows(eng, toks, prompt):
    """Logits of the prompt's last token and of every later token fed alone."""
    stream = eng.begin_stream(torch.tensor([toks[:prompt]], device="cuda"), None, max_length=len(toks) + 2, eos_token_id=-1)
    rows = [stream.logits()[0].clone()]
    for t in toks[prompt:]:
        stream.step(feed([t]))
        rows.append(stream.logits()[0].clone())
    stream.close()
    return torch.stack(rows)


# ------------------------------------------------------------------------------------------ kernels alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,W", [(1, 72), (5, 1100), (8, 4104), (3, 50), (70, 72), (40, 2052), (9, 131), (2, 17000)])
def test_norm_on_the_way_back(dtype, rows, W):
    """x + norm(c1 (y1 + b) + c2 y2) w with and without the second part and the bias, on the vector and the scalar path, for few and
    for many rows; the copy handed to the next sublayer is the updated stream."""
    g = torch.Generator().manual_seed(rows * W)
    x, y1, y2 = (torch.randn(rows, W, generator=g) * 2 for _ in range(3))
    w, b = ((torch.randn(W, generator=g) * 0.5 + c).to(torch.bfloat16) for c in (1.0, 0.0))
    eps = 0.3
    for bias, c1, second, c2 in ((None, 1.0, False, 0.0), (b, 0.6, True, -1.3), (None, -0.2, True, 0.9), (b, 2.0, False, 0.0)):
        y = c1 * (y1.double() + (bias.double() if bias is not None else 0)) + (c2 * y2.double() if second else 0)
        want = x.double() + O.rms_norm(y, w.double(), eps)
        xd = x.cuda().clone()
        dev = lambda t: t.cuda().to(dtype) if t is not None else None
        h = SK.postnorm_cast(y1.cuda(), dev(w), xd, eps, bias=dev(bias), c1=c1, y2=y2.cuda() if second else None, c2=c2)
        assert (xd.double().cpu() - want).abs().max() < 1e-4
        assert torch.equal(h, xd if dtype == torch.float32 else xd.to(dtype))
        s = SK.weighted_sum2(y1.cuda(), dev(bias), c1, y2.cuda() if second else None, c2)
        assert (s.double().cpu() - y).abs().max() < 1e-4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows,N", [(1, 48), (33, 50), (6, 2056)])
def test_norm_over_all_heads_with_a_gate(dtype, rows, N):
    g = torch.Generator().manual_seed(N)
    o, y = torch.randn(rows, N, generator=g), torch.randn(rows, N + 12, generator=g)
    w = (1 + 0.3 * torch.randn(N, generator=g)).to(torch.bfloat16)
    gate = y[:, 4:4 + N]
    want = O.rms_norm(o.double(), w.double(), 0.2) * torch.sigmoid(gate.double())
    got = SK.rownorm_gate(o.cuda(), w.cuda().to(dtype), y.cuda()[:, 4:4 + N], 0.2)
    assert (got.double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 3e-2)


def _scan_cells(y, H, D, Dv, offs, ib, fb, cap):
    """The oracle's matrix memory over the projection rows y [T, n] of one sequence."""
    T = y.shape[0]
    y = y.double()
    q, k, v, i, f = (y[:, o:o + n] for o, n in zip(offs, (H * D, H * D, H * Dv, H, H)))
    i = cap * torch.tanh((i + ib.double()) / cap)
    f = O.log_sigmoid(cap * torch.tanh((f + fb.double()) / cap))
    return O.mlstm_cell(q.reshape(T, H, D) * D ** -0.5, k.reshape(T, H, D), v.reshape(T, H, Dv), i, f)


@pytest.mark.parametrize("H,D,Dv,cap", [(2, 24, 20, 6.0), (1, 70, 33, 15.0), (3, 5, 1, 2.0), (2, 264, 6, 4.0), (1, 32, 128, 8.0)])
@pytest.mark.parametrize("cuts", [[1, 1, 1, 5, 8, 3], [9, 40, 2], [300], [2, 520, 1, 7], [1200]])
def test_matrix_memory_alone(H, D, Dv, cap, cuts):
    """Read-outs before the head norm (which would hide the denominator) for two rows, one left-padded, fed in portions: fused
    launches, prompts, prompts long enough to be cut into chunks of time, and the running maximum across all of them.  Input gates
    range from e^-cap to e^cap, so the maximum jumps, decays and stays below its start at 0."""
    T, n = sum(cuts), 2 * H * D + H * Dv + 2 * H
    offs = (4, 4 + H * D, 4 + 2 * H * D, 4 + 2 * H * D + H * Dv, 4 + 2 * H * D + H * Dv + H)
    g = torch.Generator().manual_seed(H * D + T)
    y = torch.randn(2, T, n + 8, generator=g)
    y[:, :, offs[3]:offs[3] + H] = y[:, :, offs[3]:offs[3] + H] * 4.0 - 4.0
    y[:, :, offs[4]:offs[4] + H] += 3.0
    if T > 20:
        y[:, T // 2:, offs[4]:offs[4] + H] += 12.0                        # a stretch that keeps almost everything
        y[:, 2 * T // 3, offs[3]:offs[3] + H] = 40.0                      # one token whose input gate is at the cap
    ib, fb = (torch.randn(H, generator=g).to(torch.bfloat16) for _ in range(2))
    first = [0, min(3, cuts[0] - 1)]
    st, ms = torch.zeros(2, H, D, Dv + 1, device="cuda"), torch.zeros(2, H, device="cuda")
    pad, ln = i32(first), i32([0])
    got, at = [], 0
    for c in cuts:
        ln.fill_(at)
        yc = y[:, at:at + c].reshape(2 * c, n + 8).contiguous().cuda()
        o, aux = SK.mlstm_scan(yc, offs[0], offs[1], offs[2], offs[3], offs[4], ib.cuda(), fb.cuda(), cap, D ** -0.5, st, ms, ln, pad, 2, c, H,
                               D, Dv)
        o, aux = o.view(2, c, H, Dv + 1).double().cpu(), aux.view(2, c, 3, H).double().cpu()
        den = torch.maximum(o[..., Dv].abs(), aux[:, :, 2]) + 1e-6
        got.append(o[..., :Dv] / den[..., None])
        at += c
    got = torch.cat(got, 1)
    for b in range(2):
        want = _scan_cells(y[b, first[b]:], H, D, Dv, offs, ib, fb, cap)
        scale = want.abs().amax((1, 2), keepdim=True).clamp_min(1e-3)
        d = ((got[b, first[b]:] - want).abs() / scale).flatten(1).amax(-1)
        # a read-out whose denominator almost vanishes magnifies rounding: all but a few tokens are held to the tight bound
        assert float(d.max()) < 2e-2 and float((d > 5e-4).double().mean()) < 0.02, (b, float(d.max()))


@pytest.mark.parametrize("dtype", DTYPES)
def test_division_head_norm_and_gate(dtype):
    """The denominator shows through the head norm when eps is not small: the floor exp(-m), |n q| on both signs, and the 1e-6."""
    H, V, M, eps = 3, 18, 12, 0.5
    g = torch.Generator().manual_seed(3)
    o, aux = torch.randn(M, H, V + 1, generator=g), torch.rand(M, 3 * H, generator=g) * 1.5
    o[0] *= 1e-7
    aux[0] = 0.0
    w, gate = (1 + 0.3 * torch.randn(H * V, generator=g)).to(torch.bfloat16), torch.randn(M, H * V, generator=g)
    den = torch.maximum(o[..., V].double().abs(), aux[:, 2 * H:].double()) + 1e-6
    want = (O.rms_norm(o[..., :V].double() / den[..., None], None, eps).reshape(M, H * V) * w.double() * torch.sigmoid(gate.double()))
    got = SK.mlstm_finish(o.reshape(M, -1).cuda(), aux.cuda(), w.cuda().to(dtype), gate.cuda(), H, V, eps)
    assert (got.double().cpu() - want).abs().max() < (1e-5 if dtype == torch.float32 else 3e-2)


@pytest.mark.parametrize("H,D,Dv", [(3, 10, 14), (1, 64, 128), (2, 33, 5)])
@pytest.mark.parametrize("cuts", [[1, 8, 2], [9, 30], [3, 700]])
def test_activated_linear_attention_alone(H, D, Dv, cuts):
    T, n = sum(cuts), 2 * H * D + H * Dv
    g = torch.Generator().manual_seed(T + D)
    y = torch.randn(2, T, n, generator=g)
    decay = torch.tensor([0.9 ** (h + 1) if h else 0.9995 for h in range(H)])
    st, pad, ln = torch.zeros(2, H, D, Dv, device="cuda"), i32([0, min(2, cuts[0] - 1)]), i32([0])
    got, at = [], 0
    for c in cuts:
        ln.fill_(at)
        o = SK.activated_scan(y[:, at:at + c].reshape(2 * c, n).contiguous().cuda(), 0, H * D, 2 * H * D, decay.cuda(), SK.ACT_SILU, st, ln, pad,
                              2, c, H, D, Dv)
        got.append(o.view(2, c, H, Dv).double().cpu())
        at += c
    got = torch.cat(got, 1)
    for b, f in enumerate((0, min(2, cuts[0] - 1))):
        q, k, v = (O.silu(y[b, f:, a:a + m].double()).reshape(T - f, H, -1) for a, m in ((0, H * D), (H * D, H * D), (2 * H * D, H * Dv)))
        S, want = torch.zeros(H, D, Dv, dtype=F64), torch.zeros(T - f, H, Dv, dtype=F64)
        for s in range(T - f):
            S = decay.double()[:, None, None] * S + k[s][:, :, None] * v[s][:, None, :]
            want[s] = (q[s][:, :, None] * S).sum(1)
        assert (got[b, f:] - want).abs().max() < 1e-4 * want.abs().max()


@pytest.mark.parametrize("taps", [1, 2, 4, 9, 20])
def test_convolution_with_a_projection_bias(taps):
    """The bias is part of every projected value and of the kept state, but not of the zeros before the start (left padding too)."""
    C, cuts, first = 13, [2, 1, 30, 1, 70], [0, 1]
    T = sum(cuts)
    g = torch.Generator().manual_seed(taps)
    y, w = torch.randn(2, T, C + 5, generator=g), torch.randn(C, taps, generator=g).to(torch.bfloat16)
    bias = torch.randn(C, generator=g) * 3.0
    st = torch.zeros(2, max(taps - 1, 1), C, device="cuda")
    pad, ln, at, got = i32(first), i32([0]), 0, []
    for c in cuts:
        ln.fill_(at)
        o = SK.causal_conv(y[:, at:at + c].reshape(2 * c, C + 5).contiguous().cuda(), 3, w.cuda(), None, st, ln, pad, 2, c, act=SK.ACT_NONE,
                           in_bias=bias.cuda())
        got.append(o.view(2, c, C).double().cpu())
        at += c
    got = torch.cat(got, 1)
    for b, f in enumerate(first):
        want = O.causal_conv(y[b, f:, 3:3 + C].double() + bias.double(), w.double())
        assert (got[b, f:] - want).abs().max() < 1e-4


# ------------------------------------------------------------------------------------------ mechanisms alone, as models
SINGLE = {
    "attention": [att()],
    "attention_plain_rotation": [att(scaling=None, rot=16, window=0)],
    "attention_unrotated": [att(rot=0)],
    "attention_uncapped": [att(cap=0.0, scale=0.8)],
    "attention_hard_cap": [att(cap=0.7, scale=2.0)],
    "attention_one_value_head": [att(heads=4, kv_heads=1, dim=8, vdim=32, window=5)],
    "attention_window_of_one": [att(window=1)],
    "attention_three_heads_odd_sizes": [att(heads=3, kv_heads=3, dim=7, vdim=5, window=64, rot=6)],
    "rotation_of_two_channels": [att(heads=3, kv_heads=1, dim=10, vdim=6, rot=2, base=3.0, scaling=None)],
    "seventeen_query_heads_per_value_head": [att(heads=34, kv_heads=2, dim=8, vdim=8, window=50, rot=4)],
    "value_rows_of_320_channels": [att(heads=2, kv_heads=1, dim=16, vdim=320, window=40, rot=16)],
    "keys_of_264_channels": [att(heads=2, kv_heads=2, dim=264, vdim=8, window=0, rot=100, scale=0.06)],
    "values_mixed_in_two_later_layers": [att(), att(mix=False), att(heads=2, dim=8), att(heads=6, rot=16)],
    "first_mixing_layer_is_not_the_first": [att(mix=False, kv_heads=1, vdim=9), mem(), att(), att(heads=2, window=3)],
    "attention_and_dense": [att(mlp=dense(17))],
    "parallel": [par()],
    "parallel_without_convolution_reach": [par(conv=1)],
    "parallel_many_taps": [par(conv=11)],
    "parallel_two_taps_one_key_head": [par(heads=6, kv_heads=1, conv=2, dim=9, rot=0, window=0)],
    "parallel_scaled_rotation": [par(rot=12, scaling=SCALING, base=20.0)],
    "parallel_right_heads_differ": [par(heads=2, kv_heads=2, right=(5, 6, 22), ls=-0.3, rs=1.7, decay=[0.2, 0.5, 0.9, 0.99, 1.0])],
    "parallel_left_only": [par(ls=1.0, rs=0.0)],
    "parallel_right_only": [par(ls=0.0, rs=2.0)],
    "parallel_and_dense": [par(mlp=dense())],
    "memory": [mem()],
    "memory_one_head": [mem(heads=1, dim=40, vdim=33, cap=3.0)],
    "memory_small_values": [mem(heads=5, dim=8, vdim=2)],
    "memory_keys_of_264_channels": [mem(heads=1, dim=264, vdim=12)],
    "memory_and_dense": [mem(mlp=dense(9))],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_single_mechanism_models(dtype, name):
    cfg = config(SINGLE[name], eps=1e-2)                                  # an eps that shows where it stands in every norm
    eng, cpu = build(cfg, dtype, seed=3)
    toks = tokens(75, cfg.vocab_size, 9)
    want = oracle_logits(cfg, cpu, toks)
    got = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(got, want) < tol(dtype, cfg)
    assert err(decode_rows(eng, toks, 70), want[69:]) < tol(dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_after_every_layer(dtype):
    cfg = config(MIXED)
    eng, cpu = build(cfg, dtype, seed=4)
    toks = tokens(50, cfg.vocab_size, 11)
    want_streams = []
    want = oracle_logits(cfg, cpu, toks, want_streams)
    eng.capture_streams = []
    got = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    streams, eng.capture_streams = eng.capture_streams, None
    assert len(streams) == len(want_streams) == len(cfg.layers)
    for a, b in zip(streams, want_streams):
        assert (a.double().cpu() - b).pow(2).mean().sqrt() < (1e-4 if dtype == torch.float32 else 6e-2) * b.pow(2).mean().sqrt()
    assert err(got, want) < tol(dtype, cfg)


def test_other_constants():
    """Another eps, base, scale, interpolation, caps and width; vocabulary and width that fit no vector width."""
    layers = [att(heads=2, kv_heads=1, dim=24, vdim=16, window=11, scale=0.07, cap=0.3, rot=20, base=31.0,
                  scaling={"factor": 2.5, "low": 0.5, "high": 6.0, "original": 16}, mlp=dense(ff=17)),
              par(heads=5, kv_heads=5, dim=6, window=3, conv=5, rot=2, base=2.0, right=(2, 3, 4), ls=1.9, rs=-0.8),
              mem(heads=2, dim=3, vdim=7, cap=1.5, mlp=dense(ff=3))]
    cfg = config(layers, vocab=41, width=50, eps=3e-3)
    eng, cpu = build(cfg, torch.float32, seed=2)
    toks = tokens(60, cfg.vocab_size, 1)
    want = oracle_logits(cfg, cpu, toks)
    assert err(eng.forward(torch.tensor([toks], device="cuda")).logits[0], want) < TOL[torch.float32]
    assert err(decode_rows(eng, toks, 3), want[2:]) < TOL[torch.float32]


# ------------------------------------------------------------------------------------------ decoding, portions, batches
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [1, 2, 31, 33])
def test_decode_matches_prefill_and_oracle(dtype, prompt):
    cfg = config(MIXED)
    eng, cpu = build(cfg, dtype, seed=7)
    toks = tokens(prompt + 45, cfg.vocab_size, 13)
    want = oracle_logits(cfg, cpu, toks)
    whole = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(whole, want) < tol(dtype, cfg)
    rows = decode_rows(eng, toks, prompt)
    assert err(rows, want[prompt - 1:]) < tol(dtype, cfg)
    assert err(rows, whole[prompt - 1:]) < tol(dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(dtype):
    """Three hundred tokens decoded one by one after a two-token prompt, windows passing over decoded tokens."""
    cfg = config([mem(), att(window=37, mlp=dense()), par(window=64), att(window=100)])
    eng, cpu = build(cfg, dtype, seed=21)
    toks = tokens(302, cfg.vocab_size, 5)
    assert err(decode_rows(eng, toks, 2), oracle_logits(cfg, cpu, toks)[1:]) < tol(dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2, 2, 2, 30], [33, 2, 9], [5, 64, 3], [1, 2, 200], [2] * 12])
def test_prompt_in_portions(dtype, cuts):
    """The same prompt fed to one cache in portions of several sizes, down to two tokens (and one): keys, convolution inputs, both
    recurrent states and the running maximum are carried from portion to portion."""
    cfg = config(MIXED)
    eng, cpu = build(cfg, dtype, seed=14)
    toks = tokens(sum(cuts), cfg.vocab_size, 31)
    want = oracle_logits(cfg, cpu, toks)
    cache = eng.new_cache(1, len(toks) + 2)
    cache.set_index(0)
    got, at = [], 0
    for n in cuts:
        got.append(eng.forward(torch.tensor([toks[at:at + n]], device="cuda"), cache=cache).logits[0])
        at += n
    assert err(torch.cat(got), want) < tol(dtype, cfg)
    assert not cache.step_values


def run_unequal_batch(cfg, dtype, lens, extra, seed):
    """Left-padded batch of prompts of the given lengths, then `extra` tokens decoded together; every row is compared with
    the oracle run of that request alone."""
    eng, cpu = build(cfg, dtype, seed=seed)
    seqs = [tokens(n + extra, cfg.vocab_size, 20 + n + 100 * b) for b, n in enumerate(lens)]
    S, B = max(lens), len(lens)
    ids = torch.zeros((B, S), dtype=torch.long)
    mask = torch.zeros((B, S), dtype=torch.int32)
    rows = []
    for b, (n, s) in enumerate(zip(lens, seqs)):
        ids[b, S - n:] = torch.tensor(s[:n])
        mask[b, S - n:] = 1
        rows += [b * S + S - n + j for j in range(n)]
    stream = eng.begin_stream(ids.cuda(), mask.cuda(), max_length=S + extra + 1, eos_token_id=-1, logit_rows=torch.tensor(rows))
    got_prompt = stream.prompt_logits().clone()
    steps = []
    for j in range(extra):
        stream.step(feed([s[n + j] for n, s in zip(lens, seqs)]))
        steps.append(stream.logits().clone())
    stream.close()
    at = 0
    for b, (n, s) in enumerate(zip(lens, seqs)):
        want = oracle_logits(cfg, cpu, s)
        assert err(got_prompt[at:at + n], want[:n]) < tol(dtype, cfg), b
        assert err(torch.stack([x[b] for x in steps]), want[n:]) < tol(dtype, cfg), b
        at += n


@pytest.mark.parametrize("dtype", DTYPES)
def test_unequal_batch_equals_each_alone(dtype):
    """Prompts of 1, 7 and 40 tokens in one batch: padding must touch neither the positions, the windows, the convolution's zeros,
    the recurrent states nor the running maximum of the real tokens."""
    run_unequal_batch(config(MIXED), dtype, [1, 7, 40], 36, seed=6)


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes_and_a_batch_of_twenty(dtype):
    """Sizes that fit no vector width or tile in a batch of twenty unequal requests: more rows than the weight-streaming kernel and
    the two-stream form of the parallel mixer take.  A memory of one head whose read-out almost vanishes has no direction left that
    rounding would keep, and the head norm blows it up: in bfloat16 a larger eps keeps such tokens comparable."""
    layers = [att(heads=3, kv_heads=3, dim=10, vdim=14, window=9, rot=6, mlp=dense(ff=11)),
              par(heads=3, kv_heads=1, dim=10, conv=4, right=(1, 5, 7), mlp=dense(ff=6)), mem(heads=1, dim=9, vdim=11),
              att(heads=3, kv_heads=3, dim=6, vdim=14, window=4, rot=2)]
    run_unequal_batch(config(layers, vocab=77, width=90, eps=0.3 if dtype == torch.bfloat16 else 1e-5), dtype, [3, 17, 1, 9, 30, 2, 12, 25, 8, 21, 4, 5, 6, 7, 11, 13, 14, 15, 16, 29], 12,
                      seed=17)


def test_realistic_head_sizes():
    """128- and 64-wide heads, eight query heads per key/value head, feed-forward on the tensor cores."""
    layers = [mem(heads=4, dim=64, vdim=128, mlp=dense(ff=256)),
              att(heads=8, kv_heads=1, dim=128, vdim=128, window=96, rot=64, scale=0.09, mlp=dense(ff=256)),
              par(heads=4, kv_heads=2, dim=64, window=70, conv=4, rot=32, scale=0.125, right=(4, 64, 64), mlp=dense(ff=256)),
              att(heads=4, kv_heads=1, dim=64, vdim=128, window=0, rot=64, scale=0.125)]
    run_unequal_batch(config(layers, width=256, vocab=128), torch.bfloat16, [5, 150, 131], 40, seed=13)


def test_state_and_cache_are_clean_when_used_again():
    """The same decode state serves request after request: a second, shorter request must see nothing of the first (old keys
    invisible, convolution inputs and states zero, the running maximum back at 0, old left-pad counts gone)."""
    cfg = config(MIXED)
    eng, cpu = build(cfg, torch.float32, seed=8)
    a, b = tokens(50, cfg.vocab_size, 1), tokens(9, cfg.vocab_size, 2)
    pad_ids = torch.zeros((2, 50), dtype=torch.long)
    pad_ids[0] = torch.tensor(a)
    pad_ids[1, 41:] = torch.tensor(b)
    mask = (torch.arange(50)[None, :] >= torch.tensor([0, 41])[:, None]).int()
    out1 = eng.generate(pad_ids.cuda(), mask.cuda(), max_length=60, eos_token_id=-1)
    st = eng._decode_state(2, 60)
    ids2 = torch.tensor([b, b[::-1]])
    out2 = eng.generate(ids2.cuda(), None, max_length=60, eos_token_id=-1)          # same (B, max_length): same state, same cache
    assert eng._decode_state(2, 60) is st
    fresh, _ = build(cfg, torch.float32, seed=8)
    out3 = fresh.generate(ids2.cuda(), None, max_length=60, eos_token_id=-1)
    assert torch.equal(out2, out3)
    assert out1.shape == (2, 60)
    eng.release_state(st)
    assert (2, 60) not in eng._decode_states
    out4 = eng.generate(ids2.cuda(), None, max_length=60, eos_token_id=-1)
    assert torch.equal(out4, out3)


# ------------------------------------------------------------------------------------------ made-to-show inputs
A_TOK, B_TOK = 61, 60
WIDTH = 48


def _planted(kind, window, dtype, sink=0.0, cap=0.0, dim=64, vdim=None, rot=32, score=24.0, seed=5):
    """One layer of attention alone ("attention", or the left half of a "parallel" mixer with the right half scaled to nothing).
    Tokens A and B embed as unit vectors, so the layer sees one column of each projection for them: A's key lies in key/value head 0
    only and B's query in query head 0 only, the same vector on the unrotated channels.  After the norms over all heads their score
    is `score` at any distance, while a random key's has a deviation of score / sqrt(dim · kv_heads)."""
    H, G = 4, 2
    scale = score / (dim * math.sqrt(H * G))
    layer = att(heads=H, kv_heads=G, dim=dim, vdim=vdim or 12, window=window, scale=scale, cap=cap, rot=rot, base=100.0) \
        if kind == "attention" else par(heads=H, kv_heads=G, dim=dim, window=window, scale=scale, conv=3, rot=rot, rs=0.0, ls=1.5)
    cfg = config([layer], vocab=64, width=WIDTH, eps=1e-6)
    p = "l0.mix." if kind == "attention" else "l0.mix.left."

    def tweak(t):
        for tok, ch in ((B_TOK, 0), (A_TOK, 1)):
            t["embed"][tok] = 0
            t["embed"][tok, ch] = 1.0
        t[p + "q.norm"].fill_(1.0)
        t[p + "k.norm"].fill_(1.0)
        u = torch.zeros(dim, device="cuda")
        u[rot:] = torch.randn(dim - rot, device="cuda", generator=torch.Generator(device="cuda").manual_seed(3))
        for name, ch in (("q", 0), ("k", 1)):
            t[p + name][:, ch] = 0
            t[p + name][:dim, ch] = u.to(torch.bfloat16)
        if kind == "attention":
            t[p + "sink"].fill_(sink)
        else:
            for name in ("q", "k"):
                t[p + name + ".b"].zero_()
            t[p + "o.b"].zero_()
            for name in ("q", "k"):
                t[p + name + ".conv"].zero_()
                t[p + name + ".conv"][:, -1] = 1.0
    eng, cpu = build(cfg, dtype, seed=seed, tweak=tweak)
    return cfg, eng, cpu


def _check_last(cfg, eng, cpu, toks, dtype, at, matters):
    """The last token's logits in a whole prompt and decoded alone, against the oracle; `matters`: whether replacing the
    planted token (at `at`) must move them."""
    want = oracle_logits(cfg, cpu, toks)
    without = list(toks)
    without[at] = 59
    moved = err(oracle_logits(cfg, cpu, without)[-1:], want[-1:])
    assert (moved > 4 * TOL[dtype]) if matters else (moved < 1e-9), moved
    whole = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(whole[-1:], want[-1:]) < TOL[dtype]
    assert err(decode_rows(eng, toks, len(toks) - 1)[-1:], want[-1:]) < TOL[dtype]


KINDS = ["attention", "left"]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("far", [0, 1, 31, 32, 33, 63, 64, 290])
def test_one_far_key_decides(dtype, kind, far):
    """Attention without a window: the planted key stands once at position `far` among 300 random ones and B is the last
    token.  A kernel that drops or misplaces it (edges of the 32-key tiles, the first slots, hundreds back) moves the
    logits far beyond the tolerance."""
    cfg, eng, cpu = _planted(kind, 0, dtype)
    toks = [2 + (i % 50) for i in range(300)]
    toks[far] = A_TOK
    toks.append(B_TOK)
    _check_last(cfg, eng, cpu, toks, dtype, far, True)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("window", [2, 24, 32, 33, 70])
@pytest.mark.parametrize("where", ["last_inside", "first_outside", "next", "far_outside"])
def test_window_edge_decides(dtype, kind, window, where):
    """The planted key stands on the last position the window shows, one before it, right before the query, or far behind.
    Attention is all that reaches back in this model, so a key outside must not matter at all."""
    n = 200                                                                      # the query's position
    at = {"last_inside": n - window + 1, "first_outside": n - window, "next": n - 1, "far_outside": n - window - 64}[where]
    cfg, eng, cpu = _planted(kind, window, dtype)
    toks = [2 + (i % 50) for i in range(n)]
    toks[at] = A_TOK
    toks.append(B_TOK)
    _check_last(cfg, eng, cpu, toks, dtype, at, n - at < window)


@pytest.mark.parametrize("dim", [128, 64])
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("window", [0, 1, 24, 33, 64, 70, 128, 200])
@pytest.mark.parametrize("where", ["last_inside", "first_outside", "far_outside"])
def test_window_edge_decides_on_the_tensor_core_path(dim, kind, window, where):
    """The same planted key with 128- and 64-wide heads in bfloat16, where prompts run the tensor-core kernels: windows that start
    inside a key tile, three query tiles, the cap, the sink and the gate in the kernel.  Every row of the prompt is compared."""
    n, size = 300, window or 301
    at = max({"last_inside": n - size + 1, "first_outside": n - size, "far_outside": n - size - 64}[where], 0)
    at = min(at, n - 1)
    cfg, eng, cpu = _planted(kind, window, torch.bfloat16, sink=17.0, cap=30.0, dim=dim, vdim=dim, rot=dim // 2)
    mixer = eng.layers[0].mixer if kind == "attention" else eng.layers[0].mixer.sides[0]
    assert mixer._flash_masked_shape()
    toks = [2 + (i % 50) for i in range(n)]
    toks[at] = A_TOK
    toks.append(B_TOK)
    _check_last(cfg, eng, cpu, toks, torch.bfloat16, at, n - at < size)
    want = oracle_logits(cfg, cpu, toks)
    whole = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(whole, want) < TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
def test_decoded_queries_leave_the_planted_key_behind(dtype, kind):
    """The planted key is in the prompt; B is then decoded again and again: A is seen until the window has passed it."""
    window = 12
    cfg, eng, cpu = _planted(kind, window, dtype)
    toks = [2 + (i % 50) for i in range(40)] + [A_TOK] + [B_TOK] * 20            # A at 40: seen up to position 51
    want = oracle_logits(cfg, cpu, toks)
    other = list(toks)
    other[40] = 59
    moved = [err(a[None], b[None]) for a, b in zip(oracle_logits(cfg, cpu, other), want)]
    assert all(m > 4 * TOL[dtype] for m in moved[41:52]) and all(m < 1e-9 for m in moved[52:])
    assert err(decode_rows(eng, toks, 41), want[40:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cap,sink", [(0.0, -30.0), (0.0, 20.0), (0.0, 27.0), (0.0, 60.0), (10.0, 9.0), (10.0, 60.0), (30.0, 20.0)])
def test_the_sink_takes_the_weight_of_the_planted_key(dtype, cap, sink):
    """A sink logit far below the planted score changes nothing, one near it shares the weight, one far above takes all of it: the
    logit is a number of its own, not scaled, not capped, and counts once; the planted score is capped."""
    cfg, eng, cpu = _planted("attention", 0, dtype, sink=sink, cap=cap)
    toks = [2 + (i % 50) for i in range(90)]
    toks[17] = A_TOK
    toks.append(B_TOK)
    want = oracle_logits(cfg, cpu, toks)
    whole = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(whole, want) < TOL[dtype]
    assert err(decode_rows(eng, toks, 90)[-1:], want[-1:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["memory", "right"])
@pytest.mark.parametrize("far", [0, 1, 7, 8, 63, 64, 65, 400])
def test_one_far_token_stays_in_the_state(dtype, kind, far):
    """A recurrent layer alone that forgets almost nothing and takes in almost nothing but token A, which comes once: it decides the
    last token's logits, in prompts (fused and chunked scans), decoded alone, and when the prompt comes in portions."""
    H, D, Dv = 2, 16, 20
    layer = mem(heads=H, dim=D, vdim=Dv, cap=14.0) if kind == "memory" else par(right=(H, D, Dv), ls=0.0, rs=1.0, decay=[0.9999, 1.0])
    cfg = config([layer], vocab=64, width=WIDTH)

    def tweak(t):
        t["embed"][A_TOK] = 0
        t["embed"][A_TOK, 1] = 1.0
        t["embed"][:A_TOK, 1] = 0.0
        if kind == "memory":
            t["l0.mix.i"].zero_()
            t["l0.mix.f"].zero_()
            t["l0.mix.i"][:, 1] = 10.0
            t["l0.mix.i.b"].fill_(-4.0)
            t["l0.mix.f.b"].fill_(13.0)
        else:
            for n in ("k", "v"):
                t["l0.mix.right." + n][:, 1] = 12.0 * torch.randn(t["l0.mix.right." + n].shape[0], device="cuda",
                                                                  generator=torch.Generator(device="cuda").manual_seed(2))
            t["l0.mix.right.k"][:, 2:] *= 0.2
            t["l0.mix.right.k"][:, 0] *= 0.2
    eng, cpu = build(cfg, dtype, seed=5, tweak=tweak)
    toks = [2 + (i % 50) for i in range(450)]
    toks[far] = A_TOK
    _check_last(cfg, eng, cpu, toks, dtype, far, True)
    want = oracle_logits(cfg, cpu, toks)
    cache = eng.new_cache(1, len(toks))
    cache.set_index(0)
    cuts, at, got = [8, 1, 56, 2, 150, 233], 0, []
    for n in cuts:
        got.append(eng.forward(torch.tensor([toks[at:at + n]], device="cuda"), cache=cache).logits[0])
        at += n
    assert err(torch.cat(got)[-1:], want[-1:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_values_reach_later_layers_of_the_same_token_only(dtype):
    """With a mixing weight of one the later layer attends to the first layer's values alone (and its own value projection is without
    effect), in prompts, portions and decoding: a stale or shifted row of values would show at once."""
    cfg = config([att(window=0), mem(), att(heads=2, dim=8, window=6)])

    def tweak(t):
        t["l2.mix.vmix"].fill_(1.0)
        t["l0.mix.vmix"].fill_(7.0)                                      # the first layer's own weight is not used
    eng, cpu = build(cfg, dtype, seed=9, tweak=tweak)
    toks = tokens(40, cfg.vocab_size, 3)
    want = oracle_logits(cfg, cpu, toks)
    free = dict(cpu)
    free["l2.mix.v"] = torch.randn_like(cpu["l2.mix.v"].float())
    assert err(oracle_logits(cfg, free, toks), want) < 1e-9
    assert err(eng.forward(torch.tensor([toks], device="cuda")).logits[0], want) < TOL[dtype]
    assert err(decode_rows(eng, toks, 5), want[4:]) < TOL[dtype]


# ------------------------------------------------------------------------------------------ the framework's entry points
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_front_end(dtype, tmp_path):
    """save_pretrained → registry → `LLaMA.generate_from_str` (left-padded batch, scheduler, on-device arg-max): every
    generated token is the oracle's arg-max given its prefix, up to near-ties."""
    from jax_llama_b200.models import registry

    cfg = config(MIXED, vocab=80)
    model = KetolixForCausalLM(cfg, dtype=dtype, seed=12, _do_init=True)
    model.save_pretrained(str(tmp_path))
    assert registry.resolve(str(tmp_path))[0] == "ketolix"
    loaded = registry.load_pretrained(str(tmp_path), dtype=dtype, device="cuda")
    assert isinstance(loaded, KetolixForCausalLM) and loaded.config.to_dict() == cfg.to_dict()
    llm = LLaMA(loaded.params, loaded, IdTokenizer(cfg.vocab_size))
    prompts = ["7 8 9 10 11 12", "40", "3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3 3"]
    texts = llm.generate_from_str(prompts, max_gen_len=24, temperature=0.0)
    cpu = {k: v.cpu() for k, v in loaded.params.items()}
    for p, t in zip(prompts, texts):
        ids = [int(x) for x in t.split()]
        n0 = len(p.split()) + 1
        assert ids[:n0] == [1] + [int(x) for x in p.split()]
        assert len(ids) > n0
        want = oracle_logits(cfg, cpu, ids)
        for j in range(n0, len(ids)):
            row = want[j - 1]
            slack = (1e-3 if dtype == torch.float32 else 0.2) * float((row - row.mean()).pow(2).mean().sqrt())
            assert row[ids[j]] >= row.max() - slack, (p, j)
    sampled = llm.generate_from_str(prompts[:1], max_gen_len=8, temperature=0.9, top_p=0.9)
    assert len(sampled[0].split()) >= 7


def test_command_line_generates_from_a_checkpoint_directory(tmp_path):
    """examples/example.py --model_dir: registry, loader, engine, scheduler and sampler behind the command line."""
    cfg = config(MIXED, vocab=80)
    KetolixForCausalLM(cfg, seed=3, _do_init=True).save_pretrained(str(tmp_path))
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    r = subprocess.run([sys.executable, os.path.join(root, "examples", "example.py"), "--model_dir", str(tmp_path), "--prompt",
                        "7 8 9", "--prompt", "40", "--max_gen_len", "6", "--temperature", "0"], capture_output=True, text=True,
                       timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [l for l in r.stdout.splitlines() if l.strip() and not l.startswith("=")]
    assert lines[0].split()[:4] == ["1", "7", "8", "9"] and lines[1].split()[:2] == ["1", "40"]
    assert all(0 <= int(t) < 80 for l in lines[:2] for t in l.split())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_of_batches_that_come_and_go(dtype, tmp_path):
    """bin/trace_run on a saved checkpoint: a request alone, a batch of three unequal requests decoded together while its
    shorter ones end, a second batch that opens while the first is still live; every wanted row against the oracle of that
    request alone."""
    import numpy as np

    cfg = config(MIXED, vocab=80)
    model = KetolixForCausalLM(cfg, seed=5, _do_init=True)
    model.save_pretrained(str(tmp_path / "m"))
    cpu = {k: v.cpu() for k, v in model.params.items()}
    seq = {"a": tokens(30, 80, 1), "b": tokens(12, 80, 2), "c": tokens(47, 80, 3), "d": tokens(9, 80, 4), "e": tokens(26, 80, 5)}
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": seq["a"][:25], "want": [0, 24]}], "end": []}]
    for j in range(25, 30):
        steps.append({"step": len(steps), "entries": [{"id": "a", "tokens": [seq["a"][j]], "want": [0] if j % 2 else []}],
                      "end": ["a"] if j == 29 else []})
    steps.append({"step": len(steps), "entries": [{"id": "b", "tokens": seq["b"][:9], "want": [8]},
                                                   {"id": "c", "tokens": seq["c"][:41], "want": list(range(0, 41, 5))},
                                                   {"id": "d", "tokens": seq["d"][:6], "want": []}], "end": []})
    for j in range(3):
        live = [("b", 9 + j, 12), ("c", 41 + j, 47), ("d", 6 + j, 9)]
        ent = [{"id": r, "tokens": [seq[r][at]], "want": [0]} for r, at, n in live]
        steps.append({"step": len(steps), "entries": ent, "end": [r for r, at, n in live if at == n - 1]})
    steps.append({"step": len(steps), "entries": [{"id": "e", "tokens": seq["e"][:20], "want": [19]},
                                                   {"id": "a2", "tokens": seq["a"][:3], "want": [2]}], "end": ["a2"]})
    for j in range(6):
        ent = [{"id": "e", "tokens": [seq["e"][20 + j]], "want": [0]}]
        if j < 3:
            ent.insert(0, {"id": "c", "tokens": [seq["c"][44 + j]], "want": [0]})
        steps.append({"step": len(steps), "entries": ent, "end": (["c"] if j == 2 else []) + (["e"] if j == 5 else [])})
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out",
                        str(out), "--max-tokens", "128"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done ")] == [f"done {i}" for i in range(len(steps))]
    seq["a2"] = seq["a"]
    full = {k: oracle_logits(cfg, cpu, v) for k, v in seq.items()}
    at = {k: 0 for k in seq}
    bound = tol(getattr(torch, dtype), cfg)
    for s in steps:
        want = []
        for e in s["entries"]:
            want += [full[e["id"]][at[e["id"]] + w] for w in e["want"]]
            at[e["id"]] += len(e["tokens"])
        path = out / f"{s['step']}.f32"
        if not want:
            assert not path.exists()
            continue
        got = torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(len(want), 80).copy())
        assert err(got, torch.stack(want)) < bound, s["step"]
