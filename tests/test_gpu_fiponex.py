"""Fiponex on the hybrid engine against the plain float64 statement of the design (`fiponex_oracle.py`).

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

from jax_llama_b200.config import FiponexConfig, MoeMlpSpec                       # noqa: E402
from jax_llama_b200.generation import LLaMA                                       # noqa: E402
from jax_llama_b200.models.feedforward import MoeFeedForward                      # noqa: E402
from jax_llama_b200.models.fiponex import FiponexForCausalLM                      # noqa: E402
from jax_llama_b200.models.hybrid_engine import HybridEngine, random_tensors      # noqa: E402
from jax_llama_b200.ops import seq_kernels as SK                                  # noqa: E402
from jax_llama_b200.tokenizers import IdTokenizer                                 # noqa: E402

from tests import fiponex_oracle as O                                             # noqa: E402

TOL = {torch.float32: 3e-4, torch.bfloat16: 8e-2}
DTYPES = [torch.float32, torch.bfloat16]
F64 = torch.float64


def tol(dtype, cfg):
    """Rounding the operands of every layer to bfloat16 adds up along the stack: the bound grows with the layers beyond four."""
    return TOL[dtype] * (max(1.0, len(cfg.layers) / 4.0) if dtype == torch.bfloat16 else 1.0)


def dense(ff=40):
    return {"kind": "dense", "ff": ff}


def moe(experts=6, top=2, ff=24):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def att(heads=4, kv_heads=2, dim=16, vdim=12, scale=0.3, coef=0.8, every=7, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if every:
        m["q_temp"] = {"coef": coef, "every": every}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def lat(heads=4, dim=12, rot_dim=6, vdim=10, kv_rank=20, window=20, scale=0.3, base=100.0, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"dims": rot_dim, "base": base}}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def delta(heads=4, kv_heads=2, dim=16, vdim=12, conv=4, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(layers, vocab=96, width=72, eps=1e-5, scale=6.0, dtype=torch.float32):
    """With dtype bfloat16 every expert of a layer is chosen (top = experts): rounding the router's input could swap two experts
    with close scores, which says nothing about the kernels.  The choice itself is tested in float32, and in bfloat16 where both
    sides see the same rounded input."""
    layers = json.loads(json.dumps(layers))
    if dtype == torch.bfloat16:
        for l in layers:
            if l["mlp"] and l["mlp"]["kind"] == "moe":
                l["mlp"]["router"]["top"] = l["mlp"]["router"]["experts"]
    return FiponexConfig.from_dict({"architecture": "Fiponex", "vocab": vocab, "width": width, "norm": {"eps": eps},
                                    "embedding": {"scale": scale}, "layers": layers})


MIXED = [delta(mlp=dense()), att(mlp=moe()), lat(mlp=dense(24)), delta(heads=3, kv_heads=3, dim=8, vdim=20, conv=3),
         att(heads=6, kv_heads=1, dim=10, vdim=8, coef=0.3, every=16, mlp=moe(experts=4, top=1)),
         lat(heads=3, dim=8, rot_dim=4, vdim=6, kv_rank=11, window=33, base=9.0, mlp=moe(experts=5, top=3, ff=9))]


def build(cfg, dtype, seed=0, graph=True, tweak=None):
    tensors = random_tensors(cfg, "cpu", seed)                          # drawn on the CPU: the same weights everywhere
    g = torch.Generator().manual_seed(seed + 1000)

    def rnd(name, mean, std):
        tensors[name] = (mean + std * torch.randn(tensors[name].shape, generator=g)).to(torch.bfloat16)

    for name in list(tensors):
        if "norm" in name:                                               # weights around zero outside the mixers, around one inside
            rnd(name, 1.0 if ".mix." in name else 0.0, 0.3)
        if name.endswith("mix.sink"):                                    # sinks that take from nothing to most of the weight
            rnd(name, 0.0, 2.0)
        if name.endswith(("q.b", "k.b", "v.b")):
            rnd(name, 0.0, 0.5)
        if name.endswith("A_log"):                                       # heads that forget at once and heads that keep
            rnd(name, -2.0, 2.0)
        if name.endswith("dt_bias"):
            rnd(name, 0.0, 1.0)
        if ".conv" in name:
            rnd(name, 0.0, 0.6)
        if name.endswith("router"):
            tensors[name] = (tensors[name].float() * 2.0).to(torch.bfloat16)
    if tweak is not None:
        tweak(tensors)
    eng = HybridEngine(cfg, tensors, dtype=dtype, device="cuda", use_cuda_graph=graph)
    return eng, tensors


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
def test_scaled_embedding(dtype):
    table = torch.randn(40, 50, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16)
    ids = [0, 39, 7, 7, 21]
    got = SK.embed_f32(i32(ids), table.cuda().to(dtype), scale=5.75)
    assert (got.double().cpu() - table.double()[ids] * 5.75).abs().max() < 1e-5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,normed,rot", [(16, True, 0), (33, True, 0), (64, True, 8), (16, False, 0), (20, False, 10)])
@pytest.mark.parametrize("coef,every", [(0.8, 7), (-0.4, 1), (2.5, 64)])
def test_query_growth_bias_and_norm(dtype, D, normed, rot, coef, every):
    """Queries, keys and values of a left-padded row and a full one, at positions around every step of the query's factor; without
    the norm too, and on rotated heads."""
    H, G, Dv, S, T = 3, 1, 10, 70, 80
    start, pads = 3, [0, 5]
    n = (H + G) * D + G * Dv
    g = torch.Generator().manual_seed(D + every)
    y, bias = torch.randn(2 * S, n, generator=g), torch.randn(n, generator=g)
    qw, kw = ((1 + 0.3 * torch.randn(D, generator=g)).to(torch.bfloat16) for _ in range(2))
    eps = 0.05
    freq = torch.tensor([30.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F64)
    ang = torch.arange(T, dtype=F64)[:, None] * freq[None]
    cos, sin = (t.float().cuda().contiguous() if rot else torch.zeros(1, 1, device="cuda") for t in (torch.cos(ang), torch.sin(ang)))
    q_out = torch.empty(2 * S, H * D, dtype=dtype, device="cuda")
    kc, vc = torch.zeros(2, G, T, D, dtype=dtype, device="cuda"), torch.zeros(2, G, T, Dv, dtype=dtype, device="cuda")
    w = (lambda t: t.cuda().to(dtype)) if normed else (lambda t: None)
    SK.attn_prep(y.cuda(), 0, H * D, (H + G) * D, q_out, kc, vc, cos, sin, rot, False, eps, i32([start]), i32(pads), 2, S, H, G, D, Dv,
                 bias=bias.cuda(), q_norm_w=w(qw), k_norm_w=w(kw), q_growth=(coef, every))
    z = (y + bias).double().view(2, S, n)
    tight = 1e-4 if dtype == torch.float32 else 5e-2
    for b, pad in enumerate(pads):
        skip = max(0, pad - start)
        pos = torch.arange(start + skip - pad, start + S - pad)
        q, k = z[b, skip:, :H * D].reshape(-1, H, D), z[b, skip:, H * D:(H + G) * D].reshape(-1, G, D)
        if normed:
            q, k = O.rms_norm(q, qw.double(), eps), O.rms_norm(k, kw.double(), eps)
        if rot:
            full = lambda t: torch.cat([torch.zeros(int(pos[0]), *t.shape[1:], dtype=F64), t])        # rotate_pairs counts from 0
            q, k = O.rotate_pairs(full(q), rot, 30.0)[int(pos[0]):], O.rotate_pairs(full(k), rot, 30.0)[int(pos[0]):]
        factor = O.query_temperature(int(pos[-1]) + 1, {"coef": coef, "every": every})[pos]
        want = q * factor[:, None, None]
        got = q_out.view(2, S, H, D)[b, skip:].double().cpu()
        assert ((got - want).abs() / (1 + want.abs())).max() < tight
        assert ((kc[b, 0, start + skip:start + S].double().cpu() - k[:, 0]).abs() / (1 + k[:, 0].abs())).max() < tight
        assert (vc[b, 0, start + skip:start + S].double().cpu() - z[b, skip:, (H + G) * D:]).abs().max() < tight * 4


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 16, 12), (3, 1, 24, 40), (16, 1, 64, 64), (8, 2, 128, 128), (6, 2, 64, 64), (2, 2, 20, 300)])
@pytest.mark.parametrize("S", [1, 2, 75])
def test_gate_per_channel_and_sink_in_the_attention_kernels(dtype, H, G, D, Dv, S):
    """Every kernel that stores attention results (tiled prompt, split-key decoding and its merge, one-launch decoding, tensor-core
    prompts of 64- and 128-wide heads) with one gate number per channel, against the plain sum; the gate is a slice of a wider row."""
    from jax_llama_b200.ops import _lib

    T, pads, scale = 90, [0, 3], 1.5 / math.sqrt(D)
    start = T - S - 5 if S < 75 else 0
    g = torch.Generator().manual_seed(H * D + S)
    q = torch.randn(2 * S, H * D, generator=g).to(torch.bfloat16)
    k, v = (torch.randn(2, G, T, n, generator=g).to(torch.bfloat16) for n in (D, Dv))
    gate = torch.randn(2 * S, H * Dv + 16, generator=g) * 3.0
    sink = torch.randn(H, generator=g) * 2.0
    dq, dk, dv, dg, ds = q.cuda().to(dtype), k.cuda().to(dtype), v.cuda().to(dtype), gate.cuda(), sink.cuda()
    view = dg[:, 8:8 + H * Dv]
    outs = [SK.attn_masked(dq, dk, dv, i32([start]), i32(pads), 2, S, H, G, D, Dv, scale, gate=view, sink=True, sink_logit=ds)]
    if S == 1:                                                           # the same without scratch: one launch
        out = torch.empty(2, H * Dv, dtype=dtype, device="cuda")
        length, pad = i32([start]), i32(pads)
        _lib.check(_lib.lib().jl_attn_masked(
            dq.data_ptr(), dk.data_ptr(), dv.data_ptr(), out.data_ptr(), view.data_ptr(), dg.stride(0), 1, length.data_ptr(), pad.data_ptr(),
            2, S, H, G, D, Dv, T, D, Dv, 0, 0, 0, 0, 0, 0, scale, 0.0, 0, 0, 1, ds.data_ptr(), 0, 0, 0, 0, 0, SK.dtype_code(dtype),
            torch.cuda.current_stream().cuda_stream), "jl_attn_masked")
        outs.append(out)
    elif dtype == torch.bfloat16 and D == Dv and D in (64, 128):
        out = torch.empty(2 * S, H * Dv, dtype=dtype, device="cuda")
        pad = i32(pads)
        _lib.check(_lib.lib().jl_flash_prefill_masked(
            dq.data_ptr(), dk.data_ptr(), dv.data_ptr(), pad.data_ptr(), out.data_ptr(), 2, S, H, G, D, T, start, scale, 0, 1, ds.data_ptr(),
            view.data_ptr(), dg.stride(0), 1, 0, 0, 0, 0, 0.0, torch.cuda.current_stream().cuda_stream), "jl_flash_prefill_masked")
        outs.append(out)
    for b, p in enumerate(pads):
        n = start + S - p                                                # tokens of the row, the S last ones are asked
        seq = torch.zeros(n, H, D, dtype=F64)
        skip = max(0, p - start)
        seq[start + skip - p:] = q.view(2, S, H, D)[b, skip:].double()
        kv = [t[b, :, p:start + S].transpose(0, 1).double() for t in (k, v)]
        want = O.softmax_attend(seq, kv[0], kv[1], scale, sink=sink.double())[start + skip - p:].reshape(-1, H * Dv)
        want = want * torch.sigmoid(gate.view(2, S, -1)[b, skip:, 8:8 + H * Dv].double())
        for got in outs:
            d = (got.view(2, S, -1)[b, skip:].double().cpu() - want).abs().max()
            assert d < (2e-5 if dtype == torch.float32 else 3e-2), float(d)


def _delta_rows(u, y, H, G, D, Dv, b_off, a_off, bias, a_log):
    """The oracle's delta rule over the rows of one sequence."""
    T = u.shape[0]
    q, k, v = (t.double() for t in (u[:, :G * D], u[:, G * D:2 * G * D], u[:, 2 * G * D:]))
    unit = lambda t: t / torch.sqrt((t * t).sum(-1, keepdim=True) + 1e-6)
    group = torch.arange(H) * G // H
    q, k = unit(q.reshape(T, G, D))[:, group] * D ** -0.5, unit(k.reshape(T, G, D))[:, group]
    decay = torch.exp(-torch.exp(a_log.double()) * O.softplus(y[:, a_off:a_off + H].double() + bias.double()))
    return O.delta_rule(q, k, v.reshape(T, H, Dv), decay, torch.sigmoid(y[:, b_off:b_off + H].double()))


@pytest.mark.parametrize("H,G,D,Dv", [(4, 2, 16, 12), (2, 2, 5, 3), (3, 1, 70, 33), (4, 4, 64, 96), (2, 1, 130, 8), (1, 1, 300, 10),
                                      (24, 6, 48, 64)])
@pytest.mark.parametrize("cuts", [[1, 1, 1, 5, 8, 3], [9, 2, 40], [2, 35, 1, 66, 10], [301]])
def test_delta_rule_with_one_decay_per_head_alone(H, G, D, Dv, cuts):
    """Read-outs before the head norm for two rows, one left-padded, fed in portions: fused launches, prompts in blocks of four tokens
    with every remainder, stages that end inside a block's reach.  Decays range from exactly zero (a token that wipes the state) over
    tiny ones to one; keys repeat, so that what the tokens of a block do to one another matters."""
    T, nu = sum(cuts), 2 * G * D + H * Dv
    g = torch.Generator().manual_seed(H * D + T)
    u, y = torch.randn(2, T, nu, generator=g), torch.randn(2, T, 2 * H + 7, generator=g)
    u[:, 1::3, G * D:2 * G * D] = u[:, 0:1, G * D:2 * G * D] + 0.1 * u[:, 1::3, G * D:2 * G * D]
    y[:, :, :H] += 1.0                                                   # beta mostly near one
    b_off, a_off = 0, H + 3
    bias, a_log = torch.randn(H, generator=g).to(torch.bfloat16), (torch.randn(H, generator=g) - 2.0).to(torch.bfloat16)
    a_log[0] = -9.0                                                      # a head that keeps
    if T > 30:
        y[:, 14, a_off:a_off + H] = 3.0e5                                # a decay of zero inside a block ...
        y[:, 20:24, a_off:a_off + H] = 60.0                              # ... and a block of tiny ones
    first = [0, min(3, cuts[0] - 1)]
    st, pad, ln = torch.zeros(2, H, D, Dv, device="cuda"), i32(first), i32([0])
    got, at = [], 0
    for c in cuts:
        ln.fill_(at)
        o = SK.delta_head_scan(u[:, at:at + c].reshape(2 * c, nu).contiguous().cuda(), 0, G * D, 2 * G * D, G,
                               y[:, at:at + c].reshape(2 * c, -1).contiguous().cuda(), b_off, a_off, bias.cuda(), a_log.cuda(), st, ln, pad, 2, c,
                               H, D, Dv)
        got.append(o.view(2, c, H, Dv).double().cpu())
        at += c
    got = torch.cat(got, 1)
    for b in range(2):
        want = _delta_rows(u[b, first[b]:], y[b, first[b]:], H, G, D, Dv, b_off, a_off, bias, a_log)
        assert (got[b, first[b]:] - want).abs().max() < 2e-5 * max(1.0, float(want.abs().max())), b
        assert first[b] == 0 or got[b, :min(first[b], cuts[0])].abs().max() == 0


def test_relu_gated_activation():
    g = torch.Generator().manual_seed(2)
    for F in (9, 16):
        y = torch.randn(7, 2 * F + 4, generator=g)
        got = SK.glu_act(y.cuda(), 0, F + 4, F, torch.float32, kind=SK.GLU_PRODUCT, act=SK.ACT_RELU)
        assert (got.double().cpu() - y[:, :F].double().clamp(min=0) * y[:, F + 4:].double()).abs().max() < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 16, 17, 300])
@pytest.mark.parametrize("experts,top,W,ff", [(6, 2, 72, 24), (5, 5, 30, 7), (40, 3, 64, 40), (3, 1, 128, 64)])
def test_experts_alone(dtype, rows, experts, top, W, ff):
    """Router choice and experts on the same (rounded) input: weights are softmax scores over all experts, not made to sum to one; few
    rows, tile-sorted rows and the tensor-core form."""
    spec = MoeMlpSpec(experts=experts, top=top, ff=ff, act="silu", score="softmax", normalise=False, gated=True)
    g = torch.Generator().manual_seed(rows + experts)
    t = {n: (torch.randn(s, generator=g) / s[1] ** 0.5).to(torch.bfloat16) for n, s in MoeFeedForward.shapes(spec, W).items()}
    t["router"] = (t["router"].float() * 3.0).to(torch.bfloat16)
    h = torch.randn(rows, W, generator=g).to(torch.bfloat16)
    got = MoeFeedForward(spec, {n: v.cuda().to(dtype) for n, v in t.items()}).run(h.cuda().to(dtype)).double().cpu()
    want = O.moe_ff(h.double(), t, "", {"router": {"experts": experts, "top": top}})
    z = torch.softmax(h.double() @ t["router"].double().T, -1).sort(-1, descending=True).values
    clear = torch.ones(rows, dtype=torch.bool) if top == experts else (z[:, top - 1] - z[:, top]) > 1e-5
    scale = want.pow(2).mean().sqrt()
    assert clear.double().mean() > 0.9
    assert ((got - want).abs()[clear]).max() / scale < (2e-4 if dtype == torch.float32 else 6e-2)


# ------------------------------------------------------------------------------------------ mechanisms alone, as models
SINGLE = {
    "attention": [att()],
    "attention_of_constant_temperature": [att(every=0)],
    "attention_temperature_every_token": [att(coef=0.5, every=1)],
    "attention_one_value_head": [att(heads=4, kv_heads=1, dim=8, vdim=32)],
    "attention_a_key_head_per_query_head": [att(heads=3, kv_heads=3, dim=7, vdim=5)],
    "attention_seventeen_query_heads_per_value_head": [att(heads=34, kv_heads=2, dim=8, vdim=8)],
    "attention_value_rows_of_320_channels": [att(heads=2, kv_heads=1, dim=16, vdim=320)],
    "attention_keys_of_264_channels": [att(heads=2, kv_heads=2, dim=264, vdim=8, scale=0.06)],
    "attention_one_head": [att(heads=1, kv_heads=1, dim=20, vdim=20)],
    "attention_64_wide": [att(heads=6, kv_heads=2, dim=64, vdim=64, scale=0.12)],
    "attention_128_wide": [att(heads=4, kv_heads=1, dim=128, vdim=128, scale=0.08)],
    "attention_and_dense": [att(mlp=dense(17))],
    "attention_and_experts": [att(mlp=moe())],
    "latent": [lat()],
    "latent_unlimited": [lat(window=0)],
    "latent_window_of_one": [lat(window=1)],
    "latent_one_head": [lat(heads=1, dim=9, rot_dim=2, vdim=33, kv_rank=7)],
    "latent_mostly_rotated": [lat(dim=3, rot_dim=20, base=5.0, kv_rank=40)],
    "latent_many_heads": [lat(heads=20, dim=4, rot_dim=4, vdim=3, kv_rank=9, window=50)],
    "latent_rank_of_260": [lat(heads=2, kv_rank=260, window=64)],
    "latent_and_experts": [lat(mlp=moe(experts=7, top=7, ff=5))],
    "delta": [delta()],
    "delta_without_convolution_reach": [delta(conv=1)],
    "delta_many_taps": [delta(conv=11)],
    "delta_one_key_head": [delta(heads=6, kv_heads=1, dim=33, vdim=7, conv=2)],
    "delta_keys_of_264_channels": [delta(heads=1, kv_heads=1, dim=264, vdim=6)],
    "delta_wide_values": [delta(heads=2, kv_heads=1, dim=8, vdim=150)],
    "delta_and_dense": [delta(mlp=dense(9))],
    "two_layers_without_feed_forward": [delta(), lat(), att()],
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(SINGLE))
def test_single_mechanism_models(dtype, name):
    cfg = config(SINGLE[name], eps=1e-2, dtype=dtype)                    # an eps that shows where it stands in every norm
    eng, cpu = build(cfg, dtype, seed=3)
    toks = tokens(75, cfg.vocab_size, 9)
    want = oracle_logits(cfg, cpu, toks)
    got = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(got, want) < tol(dtype, cfg)
    assert err(decode_rows(eng, toks, 70), want[69:]) < tol(dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_stream_after_every_layer(dtype):
    cfg = config(MIXED, dtype=dtype)
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
    """Another eps, embedding scale, bases, temperatures and widths; vocabulary and width that fit no vector width."""
    layers = [lat(heads=5, dim=6, rot_dim=10, vdim=7, kv_rank=13, window=11, scale=0.07, base=31.0, mlp=dense(ff=17)),
              att(heads=5, kv_heads=5, dim=6, vdim=9, scale=1.1, coef=-0.2, every=3, mlp=moe(experts=3, top=2, ff=3)),
              delta(heads=2, kv_heads=1, dim=3, vdim=7, conv=5, mlp=moe(experts=9, top=4, ff=6))]
    cfg = config(layers, vocab=41, width=50, eps=3e-3, scale=0.35)
    eng, cpu = build(cfg, torch.float32, seed=2)
    toks = tokens(60, cfg.vocab_size, 1)
    want = oracle_logits(cfg, cpu, toks)
    assert err(eng.forward(torch.tensor([toks], device="cuda")).logits[0], want) < TOL[torch.float32]
    assert err(decode_rows(eng, toks, 3), want[2:]) < TOL[torch.float32]


# ------------------------------------------------------------------------------------------ decoding, portions, batches
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [1, 2, 31, 33])
def test_decode_matches_prefill_and_oracle(dtype, prompt):
    cfg = config(MIXED, dtype=dtype)
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
    cfg = config([delta(), att(every=50, mlp=dense()), lat(window=37), lat(window=100)], dtype=dtype)
    eng, cpu = build(cfg, dtype, seed=21)
    toks = tokens(302, cfg.vocab_size, 5)
    assert err(decode_rows(eng, toks, 2), oracle_logits(cfg, cpu, toks)[1:]) < tol(dtype, cfg)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [[2, 2, 2, 30], [33, 2, 9], [5, 64, 3], [1, 2, 200], [2] * 12])
def test_prompt_in_portions(dtype, cuts):
    """The same prompt fed to one cache in portions of several sizes, down to two tokens (and one): keys, latents, convolution inputs
    and the recurrent state are carried from portion to portion."""
    cfg = config(MIXED, dtype=dtype)
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
    """Prompts of 1, 7 and 40 tokens in one batch: padding must touch neither the positions, the windows, the convolution's zeros nor
    the recurrent states of the real tokens."""
    run_unequal_batch(config(MIXED, dtype=dtype), dtype, [1, 7, 40], 36, seed=6)


@pytest.mark.parametrize("dtype", DTYPES)
def test_odd_sizes_and_a_batch_of_twenty(dtype):
    """Sizes that fit no vector width or tile in a batch of twenty unequal requests: more rows than the weight-streaming kernel and
    the per-pair form of the experts take."""
    layers = [att(heads=3, kv_heads=3, dim=10, vdim=14, every=5, mlp=dense(ff=11)), lat(heads=3, dim=5, rot_dim=2, vdim=7, kv_rank=9, window=9),
              delta(heads=3, kv_heads=1, dim=9, vdim=11, conv=2, mlp=moe(experts=3, top=2, ff=6))]
    run_unequal_batch(config(layers, vocab=77, width=90, dtype=dtype), dtype,
                      [3, 17, 1, 9, 30, 2, 12, 25, 8, 21, 4, 5, 6, 7, 11, 13, 14, 15, 16, 29], 12, seed=17)


def test_realistic_head_sizes():
    """128- and 64-wide heads, prompts on the tensor-core attention kernels with the gate per channel, experts on the grouped GEMM."""
    layers = [delta(heads=4, kv_heads=2, dim=128, vdim=128, mlp=dense(ff=192)),
              att(heads=16, kv_heads=2, dim=128, vdim=128, scale=0.09, every=64, mlp=moe(experts=8, top=8, ff=96)),
              lat(heads=4, dim=128, rot_dim=64, vdim=128, kv_rank=256, window=70, scale=0.07, base=10000.0, mlp=dense(ff=192)),
              att(heads=4, kv_heads=4, dim=64, vdim=64, scale=0.125, every=40)]
    run_unequal_batch(config(layers, width=320, vocab=128), torch.bfloat16, [5, 150, 131], 40, seed=13)


def test_state_and_cache_are_clean_when_used_again():
    """The same decode state serves request after request: a second, shorter request must see nothing of the first (old keys
    and latents invisible, convolution inputs and states zero, old left-pad counts gone)."""
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


def _planted(kind, window, dtype, sink=0.0, dim=64, vdim=None, rot=16, score=24.0, seed=5, coef=0.0, every=1000, heads=4, solo=True):
    """One layer of attention alone.  Tokens A and B embed as unit vectors, so the layer sees one column of each projection for them:
    A's key and B's query are the same vector in head 0 (of key/value head 0, on the unrotated channels), scaled so that their score is
    `score` at any distance (at temperature one), while a random key's has a deviation of score / sqrt(dim).  solo: B's gates let head 0
    through and hold the other heads back."""
    if kind == "attention":
        scale = score / dim
        layer = att(heads=heads, kv_heads=2, dim=dim, vdim=vdim or 12, scale=scale, coef=coef, every=every)
    else:
        scale = 0.2
        layer = lat(heads=heads, dim=dim, rot_dim=rot, vdim=vdim or 12, kv_rank=24, window=window, scale=scale)
    cfg = config([layer], vocab=64, width=WIDTH, eps=1e-6, scale=3.0)
    p = "l0.mix."

    def tweak(t):
        t["l0.norm1"].zero_()
        t["embed"][:, :2] = 0                                            # the two columns are A's and B's alone
        for tok, ch in ((B_TOK, 0), (A_TOK, 1)):
            t["embed"][tok] = 0
            t["embed"][tok, ch] = 1.0
        t[p + "sink"].fill_(sink)
        if solo:
            n = t[p + "g"].shape[0] // heads
            t[p + "g"][:n, 0], t[p + "g"][n:, 0] = 1.0, -1.0
        g = torch.Generator().manual_seed(3)
        if kind == "attention":
            u = torch.randn(dim, generator=g)
            for name, ch in (("q", 0), ("k", 1)):
                t[p + name + ".norm"].fill_(1.0)
                t[p + name + ".b"].zero_()
                t[p + name][:, ch] = torch.randn(t[p + name].shape[0], generator=g).to(torch.bfloat16)
                t[p + name][:dim, ch] = u.to(torch.bfloat16)
            t[p + "v"][:, 1] *= 3.0                                      # what A carries stands out
        else:
            c = torch.randn(24, generator=g)
            t[p + "dkv"][:24, 1] = c.to(torch.bfloat16)
            c = O.rms_norm(t[p + "dkv"][:24, 1].double(), t[p + "dkv.norm"].double(), 0.0)
            u = t[p + "uk"][:dim].double() @ c                           # A's key in head 0
            carry = torch.randn(vdim or 12, generator=g).double()
            t[p + "uv"][:vdim or 12] += (3.0 * carry[:, None] * c[None] / (c @ c)).to(torch.bfloat16)
            t[p + "q"][:dim + rot, 0] = 0
            t[p + "q"][:dim, 0] = (u * score / (scale * (u @ u) * WIDTH ** 0.5)).to(torch.bfloat16)
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


KINDS = ["attention", "latent"]


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


@pytest.mark.parametrize("dim", [128, 64])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 127, 128, 129, 299])
def test_one_far_key_decides_on_the_tensor_core_path(dim, far):
    """The same planted key with 128- and 64-wide heads in bfloat16, where prompts run the tensor-core kernels with the sink and the
    gate per channel in them.  Every row of the prompt is compared."""
    cfg, eng, cpu = _planted("attention", 0, torch.bfloat16, sink=17.0, dim=dim, vdim=dim)
    assert eng.layers[0].mixer._flash_masked_shape()
    toks = [2 + (i % 50) for i in range(300)]
    toks[far] = A_TOK
    toks.append(B_TOK)
    _check_last(cfg, eng, cpu, toks, torch.bfloat16, far, True)
    want = oracle_logits(cfg, cpu, toks)
    assert err(eng.forward(torch.tensor([toks], device="cuda")).logits[0], want) < TOL[torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [2, 24, 32, 33, 70])
@pytest.mark.parametrize("where", ["last_inside", "first_outside", "next", "far_outside"])
def test_window_edge_decides(dtype, window, where):
    """The planted key stands on the last position the window shows, one before it, right before the query, or far behind.
    Attention is all that reaches back in this model, so a key outside must not matter at all."""
    n = 200                                                                      # the query's position
    at = {"last_inside": n - window + 1, "first_outside": n - window, "next": n - 1, "far_outside": n - window - 64}[where]
    cfg, eng, cpu = _planted("latent", window, dtype)
    toks = [2 + (i % 50) for i in range(n)]
    toks[at] = A_TOK
    toks.append(B_TOK)
    _check_last(cfg, eng, cpu, toks, dtype, at, n - at < window)


@pytest.mark.parametrize("dtype", DTYPES)
def test_decoded_queries_leave_the_planted_key_behind(dtype):
    """The planted key is in the prompt; B is then decoded again and again: A is seen until the window has passed it."""
    window = 12
    cfg, eng, cpu = _planted("latent", window, dtype)
    toks = [2 + (i % 50) for i in range(40)] + [A_TOK] + [B_TOK] * 20            # A at 40: seen up to position 51
    want = oracle_logits(cfg, cpu, toks)
    other = list(toks)
    other[40] = 59
    moved = [err(a[None], b[None]) for a, b in zip(oracle_logits(cfg, cpu, other), want)]
    assert all(m > 4 * TOL[dtype] for m in moved[41:52]) and all(m < 1e-9 for m in moved[52:])
    assert err(decode_rows(eng, toks, 41), want[40:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", KINDS)
@pytest.mark.parametrize("sink", [-30.0, 20.0, 24.0, 27.0, 60.0])
def test_the_sink_takes_the_weight_of_the_planted_key(dtype, kind, sink):
    """A sink logit far below the planted score changes nothing, one near it shares the weight, one far above takes all of it: the
    logit is a number of its own, not scaled, and counts once.  (The norm after the sublayer hides a factor that all heads share: the
    other heads' sums keep their size.)"""
    cfg, eng, cpu = _planted(kind, 0, dtype, solo=False)
    cpu["l0.mix.sink"][0] = sink
    eng.layers[0].mixer.sink_logit[0] = sink
    toks = [2 + (i % 50) for i in range(90)]
    toks[17] = A_TOK
    toks.append(B_TOK)
    want = oracle_logits(cfg, cpu, toks)
    whole = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(whole, want) < TOL[dtype]
    assert err(decode_rows(eng, toks, 90)[-1:], want[-1:]) < TOL[dtype]


@pytest.mark.parametrize("every", [1, 16, 33])
def test_queries_grow_at_the_right_position(every):
    """Scores near the sink's logit and a strong growth: a factor that steps one token early or late shows, in prompts, decoded alone
    and in a left-padded batch.  A planted mistake in the oracle (a step one token late) is far outside the bound."""
    cfg, eng, cpu = _planted("attention", 0, torch.float32, score=2.0, coef=0.5, every=every, solo=False)
    cpu["l0.mix.sink"].fill_(3.0)
    eng.layers[0].mixer.sink_logit.fill_(3.0)
    toks = [A_TOK] + [B_TOK if i % 3 else 2 + (i % 50) for i in range(99)]
    want = oracle_logits(cfg, cpu, toks)
    assert err(eng.forward(torch.tensor([toks], device="cuda")).logits[0], want) < TOL[torch.float32]
    assert err(decode_rows(eng, toks, 5), want[4:]) < TOL[torch.float32]
    ids = torch.tensor([toks[:60], [0] * 23 + toks[:37]])
    mask = torch.tensor([[1] * 60, [0] * 23 + [1] * 37], dtype=torch.int32)
    out = eng.forward(ids.cuda(), attention_mask=mask.cuda()).logits
    assert err(out[0], want[:60]) < TOL[torch.float32] and err(out[1, 23:], want[:37]) < TOL[torch.float32]
    right = O.query_temperature
    try:
        O.query_temperature = lambda T, q: torch.cat([right(T, q)[:1], right(T, q)[:-1]])
        late = oracle_logits(cfg, cpu, toks)
    finally:
        O.query_temperature = right
    steps = [p for p in range(1, 100) if p % 3 != 1 and (p + 1) // every != p // every and toks[p] == B_TOK]
    assert steps and all(err(late[p:p + 1], want[p:p + 1]) > 10 * TOL[torch.float32] for p in steps[:2])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("gap", [2, 5, 7, 8, 15, 16, 17, 31, 33, 216])
def test_recurrent_state_keeps_a_far_token(dtype, gap):
    """Slow decays and a filler token that writes nothing, so the state holds only what two planted tokens wrote, `gap` steps and one
    step back.  Read-outs are normed, so one token alone would hide a wrong decay; the mix of the two shows decay^(gap-1): a state
    that is lost, reset or decayed wrongly at an edge of the scan's token blocks and stages moves the logits.  In a prompt, decoded
    token by token and in portions."""
    filler, first, second = 5, 40, 41
    cfg = config([delta(heads=2, kv_heads=2, dim=16, vdim=16, conv=1)], vocab=64, width=48)

    def tweak(t):
        t["l0.norm1"].zero_()
        t["embed"][:, 3] = -1.0                                          # the filler's channel; channel 4 belongs to the planted tokens
        t["embed"][:, 4] = 0
        t["embed"][filler] = 0
        t["embed"][filler, 3] = 1.0
        t["embed"][[first, first + 2, second], 4] = 4.0
        t["embed"][second, 3] = 0.0
        t["l0.mix.A_log"].fill_(-5.0)
        t["l0.mix.k"][:, 4] = t["l0.mix.q"][:, 3]                        # their keys lean towards the filler's query, which reads them
        t["l0.mix.v"][:, 3] = 0                                          # silu(0) = 0: the filler corrects towards nothing ...
        t["l0.mix.b"].zero_()
        t["l0.mix.b"][:, 3] = -30.0                                      # ... with beta = 0; the first token writes with 1, the second with 1/2
    eng, cpu = build(cfg, dtype, seed=7, tweak=tweak)
    n = 230
    toks = [filler] * n
    toks[n - 1 - gap], toks[n - 2] = first, second
    want = oracle_logits(cfg, cpu, toks)
    other = list(toks)
    other[n - 1 - gap] = first + 2
    assert err(oracle_logits(cfg, cpu, other)[-1:], want[-1:]) > 3 * TOL[dtype]
    got = eng.forward(torch.tensor([toks], device="cuda")).logits[0]
    assert err(got[n - 1 - gap:], want[n - 1 - gap:]) < TOL[dtype]
    assert err(decode_rows(eng, toks, 10)[n - gap - 10:], want[n - 1 - gap:]) < TOL[dtype]
    cache = eng.new_cache(1, n)
    cache.set_index(0)
    cuts, at, got = [10, 3, 100, 2, 75, 40], 0, []
    for c in cuts:
        got.append(eng.forward(torch.tensor([toks[at:at + c]], device="cuda"), cache=cache).logits[0])
        at += c
    assert err(torch.cat(got)[n - 1 - gap:], want[n - 1 - gap:]) < TOL[dtype]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "latent", "delta"])
def test_first_tokens_of_a_sequence(dtype, kind):
    """Requests of one, two and three tokens alone and as the tail of a left-padded batch."""
    layer = {"attention": att(every=2), "latent": lat(window=2), "delta": delta(conv=3)}[kind]
    run_unequal_batch(config([layer], dtype=dtype), dtype, [1, 2, 3, 11], 5, seed=19)
    cfg = config([layer], dtype=dtype)
    eng, cpu = build(cfg, dtype, seed=19)
    for n in (1, 2, 3):
        toks = tokens(n, cfg.vocab_size, n)
        assert err(eng.forward(torch.tensor([toks], device="cuda")).logits[0], oracle_logits(cfg, cpu, toks)) < TOL[dtype]


# ------------------------------------------------------------------------------------------ the framework's entry points
@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_through_the_front_end(dtype, tmp_path):
    """save_pretrained → registry → `LLaMA.generate_from_str` (left-padded batch, scheduler, on-device arg-max): every
    generated token is the oracle's arg-max given its prefix, up to near-ties."""
    from jax_llama_b200.models import registry

    cfg = config(MIXED, vocab=80, dtype=dtype)
    model = FiponexForCausalLM(cfg, dtype=dtype, seed=12, _do_init=True)
    model.save_pretrained(str(tmp_path))
    assert registry.resolve(str(tmp_path))[0] == "fiponex"
    loaded = registry.load_pretrained(str(tmp_path), dtype=dtype, device="cuda")
    assert isinstance(loaded, FiponexForCausalLM) and loaded.config.to_dict() == cfg.to_dict()
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
    FiponexForCausalLM(cfg, seed=3, _do_init=True).save_pretrained(str(tmp_path))
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

    cfg = config(MIXED, vocab=80, dtype=getattr(torch, dtype))
    model = FiponexForCausalLM(cfg, seed=5, _do_init=True)
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
