"""Plain float64 statement of the Ketolix decoder, one function per mechanism, for one sequence at a time.

Nothing here imports the package: the functions take the checkpoint's tensors (name -> tensor) and the configuration as
the dictionary ``config.json`` holds, and recompute every token from the whole prefix (no cache, no state carried over).

Notation: T tokens, W model width.  Linear weights are [out, in].

  embedding      x_t = E[tok_t]
  layer          x <- x + N1(mixer(x));  x <- x + N2(ff(x))     N: RMS norm with a weight, on the way back only
  "attention"    softmax attention: q and k normed over all their channels together, rotation of neighbouring channel pairs
                 with slowed long wavelengths, capped scores, a window, a learned sink logit, values mixed with those of the
                 first layer that mixes
  "parallel"     a * left(x) + b * right(x)
     left        softmax attention whose q and k pass a short causal convolution; the values are the convolved keys
     right       linear attention with one fixed decay per head over silu-activated q, k, v
  "mlstm"        matrix memory with exponential input gate, kept in range by a running maximum
  feed-forward   down(silu(gate x) * (up x))
  output         N(x), logits against the embedding table
"""
import math

import torch

F64 = torch.float64


def rms_norm(x, w, eps):
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def log_sigmoid(z):
    return torch.where(z >= 0, -torch.log1p(torch.exp(-z.abs())), z - torch.log1p(torch.exp(-z.abs())))


def causal_conv(x, w):
    """x [T, C], w [C, taps] (last column multiplies the current token), zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    xp = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x], 0)
    y = torch.zeros_like(x)
    for j in range(taps):
        y = y + xp[j:j + T] * w[:, j]
    return y


def frequencies(dims, base, scaling=None):
    """Angle per position of every channel pair.  With scaling: waves longer than original / low are slowed by factor, waves
    shorter than original / high are kept, in between the two are blended by how many waves fit into `original`."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling:
            n, lo, hi, by = (float(scaling[k]) for k in ("original", "low", "high", "factor"))
            waves = n * f / (2.0 * math.pi)
            if waves < lo:
                f = f / by
            elif waves <= hi and hi > lo:
                s = (waves - lo) / (hi - lo)
                f = (1.0 - s) * f / by + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_pairs(x, freq):
    """x [T, heads, n]: channels (2i, 2i + 1), i < len(freq), turned by position * freq[i]; the others pass."""
    n = 2 * freq.shape[0]
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * freq[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    y = x.clone()
    y[..., 0:n:2], y[..., 1:n:2] = u * c - v * s, v * c + u * s
    return y


def softmax_attend(q, k, v, m, sink=None):
    """q [T, H, D], k [T, G, D], v [T, G, Dv] -> [T, H, Dv]; m: the mixer's entry (scale, softcap, mask); sink [H] or None."""
    T, H = q.shape[:2]
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    window = int((m.get("mask") or {}).get("size") or 0)
    if window > 0:
        seen = seen & (i - j < window)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * float(m["scale"])
        if m.get("softcap"):
            s = float(m["softcap"]) * torch.tanh(s / float(m["softcap"]))
        s = s.masked_fill(~seen, -math.inf)
        mx = s.max(-1, keepdim=True).values
        if sink is not None:
            mx = torch.maximum(mx, sink[h])
        e = torch.exp(s - mx)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - mx)
        out[:, h] = (e / den) @ v[:, h // (H // G)]
    return out


def attention(x, t, p, m, eps, first_values=None):
    """Returns (result [T, W], this layer's own values [T, G * Dv] before mixing)."""
    T = x.shape[0]
    H, G, D, Dv = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["vdim"])
    g = lambda n: t[p + n].to(F64)
    q = rms_norm(x @ g("q").T, g("q.norm"), eps).view(T, H, D)
    k = rms_norm(x @ g("k").T, g("k.norm"), eps).view(T, G, D)
    own = x @ g("v").T
    v = own
    if m.get("v_mix") and first_values is not None:
        lam = g("vmix")
        v = (1.0 - lam) * own + lam * first_values
    rot = m.get("rot")
    if rot:
        f = frequencies(int(rot["dims"]), rot["base"], rot.get("scaling"))
        q, k = rotate_pairs(q, f), rotate_pairs(k, f)
    o = softmax_attend(q, k, v.view(T, G, Dv), m, g("sink"))
    return o.reshape(T, H * Dv) @ g("o").T, own


def conv_attention(x, t, p, m, eps):
    """The left half of a "parallel" mixer."""
    T = x.shape[0]
    H, G, D = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"])
    g = lambda n: t[p + n].to(F64)
    q = causal_conv(x @ g("q").T + g("q.b"), g("q.conv"))
    k = causal_conv(x @ g("k").T + g("k.b"), g("k.conv"))
    v = k.view(T, G, D)
    q, k = rms_norm(q, g("q.norm"), eps).view(T, H, D), rms_norm(k, g("k.norm"), eps).view(T, G, D)
    rot = m.get("rot")
    if rot:
        f = frequencies(int(rot["dims"]), rot["base"], rot.get("scaling"))
        q, k = rotate_pairs(q, f), rotate_pairs(k, f)
    o = softmax_attend(q, k, v, m) * torch.sigmoid(x @ g("g").T)[:, :, None]
    return o.reshape(T, H * D) @ g("o").T + g("o.b")


def lightning(x, t, p, m, eps):
    """The right half of a "parallel" mixer."""
    T = x.shape[0]
    H, D, Dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    g = lambda n: t[p + n].to(F64)
    q, k, v = (silu(x @ g(n).T).view(T, H, -1) for n in ("q", "k", "v"))
    S = torch.zeros(H, D, Dv, dtype=F64)
    decay = torch.tensor([float(a) for a in m["decay"]], dtype=F64)[:, None, None]
    o = torch.zeros(T, H, Dv, dtype=F64)
    for s in range(T):
        S = decay * S + k[s][:, :, None] * v[s][:, None, :]
        o[s] = (q[s][:, :, None] * S).sum(1)
    return (rms_norm(o.reshape(T, H * Dv), g("norm"), eps) * torch.sigmoid(x @ g("g").T)) @ g("o").T


def parallel(x, t, p, m, eps):
    return float(m["left_scale"]) * conv_attention(x, t, p + "left.", m["left"], eps) + \
        float(m["right_scale"]) * lightning(x, t, p + "right.", m["right"], eps)


def mlstm_cell(q, k, v, i, f):
    """q, k [T, H, D], v [T, H, Dv], log gates i, f [T, H] -> read-outs [T, H, Dv]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=F64)
    n = torch.zeros(H, D, dtype=F64)
    m = torch.zeros(H, dtype=F64)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for s in range(T):
        m_new = torch.maximum(f[s] + m, i[s])
        keep, take = torch.exp(f[s] + m - m_new), torch.exp(i[s] - m_new)
        S = keep[:, None, None] * S + take[:, None, None] * k[s][:, :, None] * v[s][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[s]
        m = m_new
        den = torch.maximum((n * q[s]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[s] = (q[s][:, :, None] * S).sum(1) / den[:, None]
    return out


def mlstm(x, t, p, m, eps):
    T = x.shape[0]
    H, D, Dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    cap = float(m["gate_cap"])
    g = lambda n: t[p + n].to(F64)
    q, k, v = (x @ g("q").T * D ** -0.5).view(T, H, D), (x @ g("k").T).view(T, H, D), (x @ g("v").T).view(T, H, Dv)
    i = cap * torch.tanh((x @ g("i").T + g("i.b")) / cap)
    f = log_sigmoid(cap * torch.tanh((x @ g("f").T + g("f.b")) / cap))
    o = rms_norm(mlstm_cell(q, k, v, i, f), None, eps).reshape(T, H * Dv)
    return (o * g("norm") * torch.sigmoid(x @ g("g").T)) @ g("o").T


def dense_ff(x, t, p):
    return (silu(x @ t[p + "gate"].to(F64).T) * (x @ t[p + "up"].to(F64).T)) @ t[p + "down"].to(F64).T


def forward(tokens, t, cfg, streams=None):
    """Logits [T, vocab] of a whole sequence; `streams` (a list) receives the stream after every layer."""
    eps = float(cfg["norm"]["eps"])
    x = t["embed"].to(F64)[tokens]
    first_values = None
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        if l["type"] == "attention":
            y, own = attention(x, t, p + "mix.", m, eps, first_values)
            if m.get("v_mix") and first_values is None:
                first_values = own
        elif l["type"] == "parallel":
            y = parallel(x, t, p + "mix.", m, eps)
        else:
            y = mlstm(x, t, p + "mix.", m, eps)
        x = x + rms_norm(y, t[p + "norm1"].to(F64), eps)
        if l.get("mlp"):
            x = x + rms_norm(dense_ff(x, t, p + "mlp."), t[p + "norm2"].to(F64), eps)
        if streams is not None:
            streams.append(x.clone())
    return rms_norm(x, t["final.norm"].to(F64), eps) @ t["embed"].to(F64).T
