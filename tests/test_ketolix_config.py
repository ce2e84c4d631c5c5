"""CPU-side checks of the Ketolix integration: configuration schema, registry, tensor inventory, and properties of the float64
oracle that need no device (causality, windows, frequencies, the running maximum, mixed values)."""
import json
import math

import pytest
import torch

from jax_llama_b200.config import FoliraxConfig, KetolixConfig, RotarySpec, WavelengthScaling
from jax_llama_b200.models import registry
from jax_llama_b200.models.hybrid_engine import random_tensors, tensor_shapes
from jax_llama_b200.models.mixers import rotary_frequencies
from tests import ketolix_oracle as O

SCALING = {"factor": 3.0, "low": 1.0, "high": 5.0, "original": 48}
ATT = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.3, "softcap": 7.0, "v_mix": True, "mask": {"size": 5},
       "rot": {"dims": 4, "base": 50.0, "scaling": SCALING}}
PAR = {"left_scale": 0.8, "right_scale": -0.3,
       "left": {"heads": 3, "kv_heads": 1, "dim": 6, "vdim": 6, "scale": 0.4, "conv": 3, "mask": {"size": 9}, "rot": {"dims": 2, "base": 9.0}},
       "right": {"heads": 2, "dim": 5, "vdim": 4, "decay": [0.5, 0.99]}}
MEM = {"heads": 2, "dim": 7, "vdim": 3, "gate_cap": 11.0}
LAYERS = [{"type": "mlstm", "mixer": MEM, "mlp": None}, {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 20}},
          {"type": "parallel", "mixer": PAR, "mlp": {"kind": "dense", "ff": 12}},
          {"type": "attention", "mixer": {"heads": 2, "dim": 6, "vdim": 6, "scale": 1.0, "v_mix": True}, "mlp": None}]


def cfg_dict(**over):
    d = {"architecture": "Ketolix", "vocab": 50, "width": 24, "norm": {"eps": 1e-4}, "layers": json.loads(json.dumps(LAYERS))}
    d.update(over)
    return d


def test_config_round_trip(tmp_path):
    c = KetolixConfig.from_dict(cfg_dict())
    assert c.vocab_size == 50 and c.hidden_size == 24 and c.num_hidden_layers == 4 and c.rms_norm_eps == 1e-4
    assert c.block == "post" and c.tied_head and not c.embed_norm and c.norm_offset == 0.0
    m, a, p, b = (l.mixer for l in c.layers)
    assert (m.kind, m.heads, m.dim, m.vdim, m.gate_cap) == ("mlstm", 2, 7, 3, 11.0) and c.layers[0].mlp is None
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.window, a.softcap, a.scale) == (4, 2, 8, 6, 5, 7.0, 0.3)
    assert a.qk_norm_all and a.sink and a.sink_learned and not (a.qk_norm or a.qk_unit_norm or a.head_gate or a.bias or a.out_bias)
    assert a.rot.layout == "interleaved" and a.rot.scaling == WavelengthScaling(3.0, 1.0, 5.0, 48.0)
    assert a.v_mix == "first" and b.v_mix == "mix" and b.kv_heads == 2 and b.window == 0 and b.softcap == 0.0 and b.rot is None
    l, r = p.left, p.right
    assert (p.combine, p.left_scale, p.right_scale) == ("weighted", 0.8, -0.3)
    assert (l.heads, l.kv_heads, l.conv, l.window) == (3, 1, 3, 9) and l.v_from_k and l.bias and l.out_bias and l.head_gate and l.qk_norm_all
    assert not l.sink and not l.v_mix and l.rot.scaling is None
    assert (r.kind, r.heads, r.dim, r.vdim, r.decay) == ("lightning", 2, 5, 4, [0.5, 0.99])
    f = c.layers[1].mlp
    assert f.gated and f.act == "silu" and f.ff == 20
    c.save_pretrained(str(tmp_path))
    again = KetolixConfig.from_pretrained(str(tmp_path))
    assert again.to_dict() == c.to_dict()
    assert registry.resolve(str(tmp_path))[:2] == ("ketolix", KetolixConfig)
    from jax_llama_b200.ops.build import SUBSETS
    sub = set(SUBSETS[registry.kernel_subset("ketolix")])
    assert "float32" in registry.gpu_dtypes("ketolix") and sub < set(SUBSETS["hybrid"])
    assert "gla_scan.cu" in sub and not {"moe.cu", "delta_scan.cu", "seq_token.cu", "decode_attn.cu"} & sub


def test_scaling_kinds_are_told_apart():
    base = {"dims": 8, "base": 100.0}
    assert RotarySpec.parse(None) is None and RotarySpec.parse(base).scaling is None
    assert isinstance(RotarySpec.parse(dict(base, scaling=SCALING)).scaling, WavelengthScaling)
    old = RotarySpec.parse(dict(base, scaling={"factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})).scaling
    assert not isinstance(old, WavelengthScaling) and old.fast == 8.0


def test_validation():
    for bad in (lambda d: d["layers"][1]["mixer"].update(kv_heads=3),
                lambda d: d["layers"][1]["mixer"]["rot"].update(dims=10),
                lambda d: d["layers"][1]["mixer"]["rot"].update(dims=3),
                lambda d: d["layers"][1]["mixer"].update(softcap=-1.0),
                lambda d: d["layers"][3]["mixer"].update(vdim=5),
                lambda d: d["layers"][2]["mixer"]["left"].update(vdim=5),
                lambda d: d["layers"][2]["mixer"]["right"].update(decay=[0.5]),
                lambda d: d["layers"][0]["mixer"].update(gate_cap=0.0),
                lambda d: d["layers"][0].update(type="gla"),
                lambda d: d["layers"][1]["mlp"].update(kind="moe")):
        d = cfg_dict()
        bad(d)
        with pytest.raises(ValueError):
            KetolixConfig.from_dict(d)


def test_tensor_inventory():
    shapes = tensor_shapes(KetolixConfig.from_dict(cfg_dict()))
    assert "head" not in shapes and shapes["embed"] == (50, 24) and shapes["final.norm"] == (24,)
    assert shapes["l0.norm1"] == (24,) and "l0.norm2" not in shapes and shapes["l1.norm2"] == (24,)
    assert not any("norm1b" in k or "norm2b" in k for k in shapes)
    assert shapes["l0.mix.i"] == shapes["l0.mix.f"] == (2, 24) and shapes["l0.mix.i.b"] == shapes["l0.mix.f.b"] == (2,)
    assert shapes["l0.mix.q"] == (14, 24) and shapes["l0.mix.g"] == (6, 24) and shapes["l0.mix.norm"] == (6,) and shapes["l0.mix.o"] == (24, 6)
    assert shapes["l1.mix.q.norm"] == (32,) and shapes["l1.mix.k.norm"] == (16,) and shapes["l1.mix.sink"] == (4,)
    assert shapes["l1.mix.vmix"] == () and shapes["l3.mix.vmix"] == () and "l1.mix.g" not in shapes and "l1.mix.o.b" not in shapes
    p = "l2.mix.left."
    assert shapes[p + "q.b"] == (18,) and shapes[p + "k.b"] == (6,) and shapes[p + "o.b"] == (24,) and p + "v" not in shapes
    assert shapes[p + "q.conv"] == (18, 3) and shapes[p + "k.conv"] == (6, 3) and shapes[p + "g"] == (3, 24)
    assert "l2.mix.left.out" not in shapes and "l2.mix.left.sink" not in shapes and "l2.mix.left.vmix" not in shapes
    p = "l2.mix.right."
    assert shapes[p + "q"] == shapes[p + "k"] == (10, 24) and shapes[p + "v"] == shapes[p + "g"] == (8, 24) and shapes[p + "norm"] == (8,)
    assert shapes["l2.mlp.gate"] == shapes["l2.mlp.up"] == (12, 24) and shapes["l2.mlp.down"] == (24, 12)
    d = cfg_dict()
    d["layers"][1]["mixer"]["v_mix"] = False
    c = KetolixConfig.from_dict(d)
    assert c.layers[1].mixer.v_mix == "" and c.layers[3].mixer.v_mix == "first" and "l1.mix.vmix" not in tensor_shapes(c)
    f = FoliraxConfig.from_dict({"vocab": 20, "width": 8, "layers": [{"type": "gla", "mixer": {"heads": 1, "dim": 4, "vdim": 4, "tau": 1.0}}]})
    assert "l0.norm1b" in tensor_shapes(f)


@pytest.mark.parametrize("dims,base,scaling", [(16, 100.0, SCALING), (64, 10000.0, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 512}),
                                               (6, 3.0, {"factor": 2.0, "low": 0.5, "high": 0.5, "original": 20}), (8, 40.0, None)])
def test_frequencies_agree_with_the_oracle(dims, base, scaling):
    spec = RotarySpec.parse({"dims": dims, "base": base, "scaling": scaling})
    f, mult = rotary_frequencies(dims, base, spec.scaling)
    assert mult == 1.0 and torch.allclose(f, O.frequencies(dims, base, scaling), rtol=1e-12, atol=0)
    if scaling and scaling["factor"] == 8.0:                              # all three branches occur
        plain = O.frequencies(dims, base)
        ratio = f / plain
        assert ratio[0] == 1.0 and abs(ratio[-1] - 1 / 8) < 1e-12 and ((ratio > 0.13) & (ratio < 0.99)).any()


def _random(c, seed=0):
    return {k: v.float() for k, v in random_tensors(c, "cpu", seed).items()}


def test_oracle_is_causal_and_bounded_by_its_windows():
    c = KetolixConfig.from_dict(cfg_dict())
    t = _random(c)
    toks = [3, 9, 27, 4, 11, 45, 6, 6, 30, 2, 17, 8]
    base = O.forward(toks, t, c.to_dict())
    other = list(toks)
    other[7] = 40
    moved = O.forward(other, t, c.to_dict())
    assert (base[:7] - moved[:7]).abs().max() == 0 and (base[7:] - moved[7:]).abs().max() > 1e-3
    one = cfg_dict(layers=[json.loads(json.dumps(LAYERS[1]))])
    one["layers"][0]["mixer"]["mask"]["size"] = 3
    c1 = KetolixConfig.from_dict(one)
    t1 = _random(c1, 1)
    a = O.forward(toks, t1, c1.to_dict())
    other = list(toks)
    other[4] = 40
    b = O.forward(other, t1, c1.to_dict())
    assert (a[4:7] - b[4:7]).abs().max() > 1e-4 and (a[7:] - b[7:]).abs().max() == 0


def test_oracle_convolution_window_and_state():
    """The left half of a parallel mixer reaches window - 1 + taps - 1 tokens back, the right half to the start."""
    d = cfg_dict(layers=[json.loads(json.dumps(LAYERS[2]))])
    d["layers"][0]["mixer"]["left"]["mask"]["size"] = 3
    d["layers"][0]["mlp"] = None
    for side, reach in (("left", 2 + 2), ("right", 99)):
        e = json.loads(json.dumps(d))
        e["layers"][0]["mixer"]["right_scale" if side == "left" else "left_scale"] = 0.0
        c = KetolixConfig.from_dict(e)
        t = _random(c, 2)
        toks = [3, 9, 27, 4, 11, 45, 6, 6, 30, 2, 17, 8]
        other = list(toks)
        other[2] = 40
        diff = (O.forward(toks, t, c.to_dict()) - O.forward(other, t, c.to_dict())).abs().amax(-1)
        assert all((diff[i] > 1e-9) == (2 <= i <= 2 + reach) for i in range(12)), side


def test_oracle_memory_does_not_depend_on_the_running_maximum():
    """The maximum only keeps the numbers in range: the same read-outs come from the plain sums, with the floor 1 in their units."""
    g = torch.Generator().manual_seed(4)
    T, H, D, V = 14, 2, 5, 3
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    i, f = torch.randn(T, H, generator=g, dtype=torch.float64) * 2, -torch.rand(T, H, generator=g, dtype=torch.float64)
    got = O.mlstm_cell(q, k, v, i, f)
    for t in range(T):
        w = torch.exp(i[:t + 1] + torch.cumsum(f, 0)[t] - torch.cumsum(f, 0)[:t + 1])               # [t+1, H]
        s = (k[:t + 1] * q[t]).sum(-1) * w
        m = 0.0
        for u in range(t + 1):
            m = torch.maximum(f[u] + m, i[u])
        want = torch.einsum("sh,shv->hv", s, v[:t + 1]) / (torch.clamp(s.sum(0).abs(), min=1.0) + 1e-6 * torch.exp(m))[:, None]
        assert (got[t] - want).abs().max() < 1e-9


def test_oracle_caps_and_mixes():
    x = torch.tensor([[[8.0]], [[-8.0]]], dtype=torch.float64)
    m = {"scale": 1.0, "softcap": 2.0}
    k = torch.ones(2, 1, 1, dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    sink = torch.tensor([1.5], dtype=torch.float64)
    o = O.softmax_attend(x, k, v, m, sink)
    hi, lo = 2.0 * math.tanh(4.0), -2.0 * math.tanh(4.0)
    assert abs(float(o[0]) - math.exp(hi) / (math.exp(hi) + math.exp(1.5))) < 1e-12
    assert abs(float(o[1]) - math.exp(lo) / (2 * math.exp(lo) + math.exp(1.5))) < 1e-12
