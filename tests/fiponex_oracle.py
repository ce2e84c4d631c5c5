"""Plain float64 statement of the Fiponex decoder, one function per mechanism, for one sequence at a time.

Nothing here imports the package: the functions take the checkpoint's tensors (name -> tensor) and the configuration as
the dictionary ``config.json`` holds, and recompute every token from the whole prefix (no cache, no state carried over).

Notation: T tokens, W model width.  Linear weights are [out, in].

  embedding          x_t = c E[tok_t]
  layer              x <- x + N1b(mixer(N1(x)));  x <- x + N2b(ff(N2(x)))     N: RMS norm, weight 1 + w
  "attention"        softmax attention without rotation: biased q, k, v; q and k normed per head with a weight; q scaled up
                     slowly with its position; a learned sink logit; sigmoid gate per output channel
  "latent_attention" softmax attention over a window through one normed latent per token and one rotated key part shared by
                     the heads; a learned sink logit; sigmoid gate per head
  "delta"            delta rule with one decay per head over convolved, activated, unit-length q and k
  feed-forward       down(relu(gate x) * (up x)), or a mixture of experts down(silu(gate x) * (up x)) weighted by their
                     softmax scores as they are
  output             N(x), logits against ``head``
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def block_norm(x, w, eps):
    return rms_norm(x, 1.0 + w.to(F64), eps)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def query_temperature(T, q_temp):
    """Factor on the query at positions 0 .. T-1: 1 + coef ln(1 + floor((p + 1) / every))."""
    if not q_temp:
        return torch.ones(T, dtype=F64)
    every = int(q_temp["every"])
    return torch.tensor([1.0 + float(q_temp["coef"]) * math.log(1 + (p + 1) // every) for p in range(T)], dtype=F64)


def softmax_attend(q, k, v, scale, window=0, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; sink [H] or None: one more term in every denominator."""
    T, H = q.shape[:2]
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    if window > 0:
        seen = seen & (i - j < window)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h * G // H
        s = ((q[:, h] @ k[:, g].T) * float(scale)).masked_fill(~seen, -math.inf)
        mx = s.max(-1, keepdim=True).values
        if sink is not None:
            mx = torch.maximum(mx, sink[h])
        e = torch.exp(s - mx)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - mx)
        out[:, h] = (e / den) @ v[:, g]
    return out


def attention(x, t, p, m, eps):
    T = x.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["vdim"])
    w = lambda n: t[p + n].to(F64)
    q = rms_norm((x @ w("q").T + w("q.b")).view(T, H, D), w("q.norm"), eps)
    k = rms_norm((x @ w("k").T + w("k.b")).view(T, G, D), w("k.norm"), eps)
    v = (x @ w("v").T + w("v.b")).view(T, G, Dv)
    q = q * query_temperature(T, m.get("q_temp"))[:, None, None]
    o = softmax_attend(q, k, v, m["scale"], sink=w("sink")).reshape(T, H * Dv)
    return (o * torch.sigmoid(x @ w("g").T)) @ w("o").T


def rotate_pairs(x, dims, base):
    """x [T, heads, n]: the leading `dims` channels turned in neighbouring pairs by position * base^(-2i/dims)."""
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    y = x.clone()
    y[..., 0:dims:2], y[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return y


def latent_attention(x, t, p, m, eps):
    T = x.shape[0]
    H, D, R, Dv, K = int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"])
    w = lambda n: t[p + n].to(F64)
    q = (x @ w("q").T).view(T, H, D + R)
    low = x @ w("dkv").T
    c = rms_norm(low[:, :K], w("dkv.norm"), eps)
    turn = lambda z: rotate_pairs(z, int(m["rot"]["dims"]), m["rot"]["base"])
    q = torch.cat([q[..., :D], turn(q[..., D:])], -1)
    shared = turn(low[:, None, K:])
    k = torch.cat([(c @ w("uk").T).view(T, H, D), shared.expand(T, H, R)], -1)
    v = (c @ w("uv").T).view(T, H, Dv)
    o = softmax_attend(q, k, v, m["scale"], window=int((m.get("mask") or {}).get("size") or 0), sink=w("sink"))
    return (o * torch.sigmoid(x @ w("g").T)[:, :, None]).reshape(T, H * Dv) @ w("o").T


def causal_conv(x, w):
    """x [T, C], w [C, taps] (last column multiplies the current token), zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    xp = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x], 0)
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + xp[j:j + T] * w[:, j]
    return y


def delta_rule(q, k, v, decay, beta):
    """q, k [T, H, D], v [T, H, Dv], decay, beta [T, H] -> read-outs [T, H, Dv]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for s in range(T):
        S = decay[s][:, None, None] * S
        u = beta[s][:, None] * (v[s] - (k[s][:, :, None] * S).sum(1))
        S = S + k[s][:, :, None] * u[:, None, :]
        out[s] = (q[s][:, :, None] * S).sum(1)
    return out


def delta(x, t, p, m, eps):
    T = x.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["vdim"])
    w = lambda n: t[p + n].to(F64)
    q, k, v = (silu(causal_conv(x @ w(n).T, w(n + ".conv"))) for n in ("q", "k", "v"))
    unit = lambda z: z / torch.sqrt((z * z).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q.view(T, G, D)) * D ** -0.5, unit(k.view(T, G, D))
    group = torch.arange(H) * G // H
    beta = torch.sigmoid(x @ w("b").T)
    decay = torch.exp(-torch.exp(w("A_log")) * softplus(x @ w("a").T + w("dt_bias")))
    o = rms_norm(delta_rule(q[:, group], k[:, group], v.view(T, H, Dv), decay, beta), w("norm"), eps).reshape(T, H * Dv)
    return (o * silu(x @ w("g").T)) @ w("o").T


def dense_ff(x, t, p):
    w = lambda n: t[p + n].to(F64)
    return (torch.clamp(x @ w("gate").T, min=0.0) * (x @ w("up").T)) @ w("down").T


def moe_ff(x, t, p, mlp):
    E, top = int(mlp["router"]["experts"]), int(mlp["router"]["top"])
    w = lambda n: t[p + n].to(F64)
    s = torch.softmax(x @ w("router").T, -1)
    chosen = torch.zeros_like(s).scatter(-1, s.topk(top, -1).indices, 1.0)
    y = torch.zeros_like(x)
    for e in range(E):
        z = (silu(x @ w(f"e{e}.gate").T) * (x @ w(f"e{e}.up").T)) @ w(f"e{e}.down").T
        y = y + (s * chosen)[:, e:e + 1] * z
    return y


MIXERS = {"attention": attention, "latent_attention": latent_attention, "delta": delta}


def forward(tokens, t, cfg, streams=None):
    """Logits [T, vocab] of a whole sequence; `streams` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = t["embed"].to(F64)[tokens] * float(cfg["embedding"]["scale"])
    for i, l in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = MIXERS[l["type"]](block_norm(x, t[p + "norm1"], eps), t, p + "mix.", l["mixer"], eps)
        x = x + block_norm(y, t[p + "norm1b"], eps)
        if l.get("mlp"):
            h = block_norm(x, t[p + "norm2"], eps)
            y = dense_ff(h, t, p + "mlp.") if l["mlp"].get("kind", "dense") == "dense" else moe_ff(h, t, p + "mlp.", l["mlp"])
            x = x + block_norm(y, t[p + "norm2b"], eps)
        if streams is not None:
            streams.append(x.clone())
    return block_norm(x, t["final.norm"], eps) @ t["head"].to(F64).T
