"""CPU-side checks of the Fiponex integration: configuration schema, registry, tensor inventory, and properties of the float64
oracle that need no device (causality, windows, the query's growth, the delta rule's token blocks)."""
import json
import math

import pytest
import torch

from jax_llama_b200.config import FiponexConfig, FoliraxConfig, NikonexConfig
from jax_llama_b200.models import registry
from jax_llama_b200.models.hybrid_engine import random_tensors, tensor_shapes
from jax_llama_b200.models.mixers import MIXERS, DeltaRuleMixer
from tests import fiponex_oracle as O

ATT = {"heads": 6, "kv_heads": 2, "dim": 8, "vdim": 5, "scale": 0.3, "q_temp": {"coef": 0.7, "every": 4}}
LAT = {"heads": 3, "dim": 6, "rot_dim": 4, "vdim": 7, "kv_rank": 9, "scale": 0.4, "mask": {"size": 5}, "rot": {"dims": 4, "base": 50.0}}
DEL = {"heads": 4, "kv_heads": 2, "dim": 5, "vdim": 6, "conv": 3}
MOE = {"kind": "moe", "router": {"experts": 5, "top": 2}, "expert": {"ff": 11}}
LAYERS = [{"type": "delta", "mixer": DEL, "mlp": MOE}, {"type": "attention", "mixer": ATT, "mlp": {"kind": "dense", "ff": 20}},
          {"type": "latent_attention", "mixer": LAT, "mlp": None}]
TOKS = [3, 9, 27, 4, 11, 45, 6, 6, 30, 2, 17, 8]


def cfg_dict(**over):
    d = {"architecture": "Fiponex", "vocab": 50, "width": 24, "norm": {"eps": 1e-4}, "embedding": {"scale": 2.5},
         "layers": json.loads(json.dumps(LAYERS))}
    d.update(over)
    return d


def one(layer, **mixer):
    l = json.loads(json.dumps(layer))
    l["mixer"].update(mixer)
    l["mlp"] = None
    return FiponexConfig.from_dict(cfg_dict(layers=[l]))


def _random(c, seed=0):
    return {k: v.float() for k, v in random_tensors(c, "cpu", seed).items()}


def test_config_round_trip(tmp_path):
    c = FiponexConfig.from_dict(cfg_dict())
    assert c.vocab_size == 50 and c.hidden_size == 24 and c.num_hidden_layers == 3 and c.rms_norm_eps == 1e-4
    assert c.block == "sandwich" and c.norm_offset == 1.0 and not c.tied_head and c.embedding_scale == 2.5 and c.pair_embedding is None
    d, a, l = (x.mixer for x in c.layers)
    assert (d.kind, d.heads, d.kv_heads, d.dim, d.vdim, d.conv) == ("delta", 4, 2, 5, 6, 3) and d.head_decay
    assert (a.heads, a.kv_heads, a.dim, a.vdim, a.scale, a.q_growth) == (6, 2, 8, 5, 0.3, (0.7, 4))
    assert a.bias and a.qk_norm and a.sink and a.sink_learned and a.channel_gate and a.rot is None and a.window == 0
    assert not (a.head_gate or a.qk_unit_norm or a.qk_norm_all or a.out_bias or a.v_rot or a.softcap)
    assert (l.heads, l.dim, l.rot_dim, l.vdim, l.q_rank, l.kv_rank, l.scale, l.window) == (3, 6, 4, 7, 0, 9, 0.4, 5)
    assert l.sink_learned and l.head_gate and (l.rot.dims, l.rot.base, l.rot.layout, l.rot.scaling) == (4, 50.0, "interleaved", None)
    m, f = c.layers[0].mlp, c.layers[1].mlp
    assert (m.kind, m.experts, m.top, m.ff, m.act, m.score, m.normalise, m.scale) == ("moe", 5, 2, 11, "silu", "softmax", False, 1.0)
    assert m.gated and not (m.shared_ff or m.identity or m.choice_bias or m.router_bias) and m.groups == 1
    assert (f.kind, f.ff, f.act, f.gated) == ("dense", 20, "relu", True) and c.layers[2].mlp is None
    c.save_pretrained(str(tmp_path))
    assert FiponexConfig.from_pretrained(str(tmp_path)).to_dict() == c.to_dict()
    assert registry.resolve(str(tmp_path))[:2] == ("fiponex", FiponexConfig)
    from jax_llama_b200.ops.build import SUBSETS
    sub = set(SUBSETS[registry.kernel_subset("fiponex")])
    assert "float32" in registry.gpu_dtypes("fiponex") and sub < set(SUBSETS["hybrid"])
    assert {"delta_scan.cu", "moe.cu"} < sub and not {"gla_scan.cu", "seq_token.cu", "decode_attn.cu"} & sub


def test_defaults_and_absent_branches():
    bare = {k: v for k, v in ATT.items() if k not in ("kv_heads", "q_temp")}
    c = FiponexConfig.from_dict(cfg_dict(layers=[{"type": "attention", "mixer": bare, "mlp": None}]))
    assert c.layers[0].mixer.kv_heads == 6 and c.layers[0].mixer.q_growth is None
    assert one({"type": "latent_attention", "mixer": LAT}, mask=None).layers[0].mixer.window == 0
    assert FiponexConfig.from_dict({k: v for k, v in cfg_dict().items() if k != "embedding"}).embedding_scale == 1.0
    assert MIXERS["delta"] is DeltaRuleMixer is MIXERS["channel_delta"]


def test_validation():
    for bad in (lambda d: d["layers"][0]["mixer"].update(kv_heads=3),
                lambda d: d["layers"][0]["mixer"].update(conv=0),
                lambda d: d["layers"][0]["mlp"]["router"].update(top=6),
                lambda d: d["layers"][0]["mlp"]["router"].update(top=0),
                lambda d: d["layers"][0].update(type="gla"),
                lambda d: d["layers"][1]["mixer"].update(kv_heads=4),
                lambda d: d["layers"][1]["mixer"]["q_temp"].update(every=0),
                lambda d: d["layers"][1]["mixer"]["q_temp"].update(every=2.5),
                lambda d: d["layers"][1]["mlp"].update(kind="sparse"),
                lambda d: d["layers"][2]["mixer"]["rot"].update(dims=6),
                lambda d: d["layers"][2]["mixer"]["rot"].update(dims=3),
                lambda d: d["layers"][2]["mixer"].update(rot=None),
                lambda d: d["layers"][2]["mixer"].update(kv_rank=0),
                lambda d: d["layers"][2]["mixer"]["mask"].update(size=-1)):
        d = cfg_dict()
        bad(d)
        with pytest.raises(ValueError):
            FiponexConfig.from_dict(d)


def test_tensor_inventory():
    s = tensor_shapes(FiponexConfig.from_dict(cfg_dict()))
    assert s["embed"] == s["head"] == (50, 24) and s["final.norm"] == (24,)
    assert all(s[f"l{i}.norm1"] == s[f"l{i}.norm1b"] == (24,) for i in range(3))
    assert all(f"l{i}.norm2" in s and f"l{i}.norm2b" in s for i in range(2)) and not any(k.startswith("l2.norm2") for k in s)
    p = "l0.mix."
    assert s[p + "q"] == s[p + "k"] == (10, 24) and s[p + "v"] == s[p + "g"] == (24, 24) and s[p + "o"] == (24, 24)
    assert s[p + "q.conv"] == (10, 3) and s[p + "v.conv"] == (24, 3) and s[p + "a"] == s[p + "b"] == (4, 24)
    assert s[p + "A_log"] == s[p + "dt_bias"] == (4,) and s[p + "norm"] == (6,) and p + "a1" not in s and p + "g2" not in s
    assert s["l0.mlp.router"] == (5, 24) and s["l0.mlp.e4.gate"] == s["l0.mlp.e4.up"] == (11, 24) and s["l0.mlp.e0.down"] == (24, 11)
    assert "l0.mlp.correction" not in s and "l0.mlp.router.b" not in s and not any("shared" in k for k in s)
    p = "l1.mix."
    assert s[p + "q"] == (48, 24) and s[p + "q.b"] == (48,) and s[p + "k.b"] == (16,) and s[p + "v"] == (10, 24) and s[p + "v.b"] == (10,)
    assert s[p + "q.norm"] == s[p + "k.norm"] == (8,) and s[p + "sink"] == (6,) and s[p + "g"] == (30, 24) and s[p + "o"] == (24, 30)
    assert p + "o.b" not in s and s["l1.mlp.gate"] == s["l1.mlp.up"] == (20, 24) and s["l1.mlp.down"] == (24, 20)
    p = "l2.mix."
    assert s[p + "q"] == (30, 24) and s[p + "dkv"] == (13, 24) and s[p + "dkv.norm"] == (9,) and s[p + "uk"] == (18, 9) and s[p + "uv"] == (21, 9)
    assert s[p + "sink"] == s[p + "g"][:1] == (3,) and s[p + "o"] == (24, 21) and p + "uq" not in s and p + "dq" not in s
    n = NikonexConfig.from_dict({"vocab": 9, "width": 8, "layers": [{"type": "latent_attention", "mixer": dict(LAT, q_rank=3), "mlp": None}]})
    ns = tensor_shapes(n)
    assert ns["l0.mix.dq"] == (3, 8) and ns["l0.mix.uq"] == (30, 3) and "l0.mix.sink" not in ns and "l0.mix.g" not in ns
    f = FoliraxConfig.from_dict({"vocab": 20, "width": 8, "layers": [{"type": "gla", "mixer": {"heads": 1, "dim": 4, "vdim": 4, "tau": 1.0}}]})
    assert f.embedding_scale == 1.0
    t = random_tensors(FiponexConfig.from_dict(cfg_dict()), "cpu")
    assert all(abs(float(t[k].float().mean()) - m) < 0.3 for k, m in (("l1.mix.q.norm", 1), ("l2.mix.dkv.norm", 1), ("l0.norm1b", 0), ("final.norm", 0)))


def test_oracle_is_causal_and_reaches_as_far_as_each_mixer():
    """A latent layer reaches window - 1 tokens back, attention and the delta rule to the start; nobody sees what comes later."""
    for layer, reach in ((LAYERS[2], 4), (LAYERS[1], 99), (LAYERS[0], 99)):
        c = one(layer)
        t = _random(c, 2)
        other = list(TOKS)
        other[2] = 40
        diff = (O.forward(TOKS, t, c.to_dict()) - O.forward(other, t, c.to_dict())).abs().amax(-1)
        assert all((diff[i] > 1e-9) == (2 <= i <= 2 + reach) for i in range(12)), layer["type"]


def test_query_temperature_steps():
    f = O.query_temperature(13, {"coef": 0.5, "every": 4})
    want = [1.0] * 3 + [1 + 0.5 * math.log(2)] * 4 + [1 + 0.5 * math.log(3)] * 4 + [1 + 0.5 * math.log(4)] * 2
    assert (f - torch.tensor(want, dtype=torch.float64)).abs().max() < 1e-15
    assert (O.query_temperature(5, None) == 1).all()


def test_blocks_of_tokens_give_the_same_read_outs():
    """The scalar form that prompts run in blocks (dot products with the state at the block's start, what the tokens of a block do to one
    another through their key and query products) against the token-by-token rule, with decays of zero and one among them."""
    g = torch.Generator().manual_seed(4)
    T, H, D, V, NB = 14, 2, 5, 3, 4
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (D, D, V))
    a, beta = torch.rand(T, H, generator=g, dtype=torch.float64), torch.rand(T, H, generator=g, dtype=torch.float64)
    a[5], a[6], a[9] = 0.0, 1.0, 1e-30
    want = O.delta_rule(q, k, v, a, beta)
    S = torch.zeros(H, D, V, dtype=torch.float64)
    for t0 in range(0, T, NB):
        n = min(NB, T - t0)
        A, r = torch.ones(H, dtype=torch.float64), []
        ks, qs = (torch.einsum("thd,hdv->thv", x[t0:t0 + n], S) for x in (k, q))
        for i in range(n):
            A = A * a[t0 + i]
            r = [x * a[t0 + i][:, None] for x in r]
            seen = A[:, None] * ks[i] + sum((k[t0 + i] * k[t0 + j]).sum(-1, keepdim=True) * r[j] for j in range(i))
            r.append(beta[t0 + i][:, None] * (v[t0 + i] - seen))
            o = A[:, None] * qs[i] + sum((q[t0 + i] * k[t0 + j]).sum(-1, keepdim=True) * r[j] for j in range(i + 1))
            assert (o - want[t0 + i]).abs().max() < 1e-12
        S = A[:, None, None] * S + sum(k[t0 + j][:, :, None] * r[j][:, None, :] for j in range(n))


def test_oracle_sink_scale_and_plain_expert_weights():
    x = torch.tensor([[[2.0]], [[2.0]]], dtype=torch.float64)
    k = torch.ones(2, 1, 1, dtype=torch.float64)
    v = torch.tensor([[[1.0]], [[0.0]]], dtype=torch.float64)
    o = O.softmax_attend(x, k, v, 0.5, sink=torch.tensor([1.5], dtype=torch.float64))
    assert abs(float(o[0]) - math.e / (math.e + math.exp(1.5))) < 1e-12
    assert abs(float(o[1]) - math.e / (2 * math.e + math.exp(1.5))) < 1e-12
    c = FiponexConfig.from_dict(cfg_dict())
    t = _random(c)
    h = torch.randn(7, 24, generator=torch.Generator().manual_seed(1), dtype=torch.float64)
    every = O.moe_ff(h, t, "l0.mlp.", {"router": {"experts": 5, "top": 5}})
    one_only = O.moe_ff(h, t, "l0.mlp.", {"router": {"experts": 5, "top": 1}})
    s = torch.softmax(h @ t["l0.mlp.router"].double().T, -1)
    best = s.argmax(-1)
    for i in range(7):
        e = f"l0.mlp.e{int(best[i])}."
        z = (O.silu(h[i] @ t[e + "gate"].double().T) * (h[i] @ t[e + "up"].double().T)) @ t[e + "down"].double().T
        assert (one_only[i] - s[i, best[i]] * z).abs().max() < 1e-12
    assert (every - one_only).abs().max() > 1e-3
