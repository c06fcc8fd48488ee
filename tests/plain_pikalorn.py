"""Plain, slow Pikalorn in float64 on the CPU: the oracle of the tests.  One function per
mechanism, written from the design's equations; nothing here is shared with the package.

Notation: x [T, W] the residual stream, h = N(x) what both sublayers of a layer read, p the position of
a token in its sequence (from 0).  Attention: H query heads, head sizes d (queries and keys) and dv
(values).  A delta layer's state is a matrix S [d, dv] per head.  A layer is
x <- x + (mixer(N(x)) + ffn(N(x))) with an RMS norm N."""
import math

import torch

F = torch.float64


def rms(x, eps, w=None):
    """x / sqrt(mean(x^2) + eps) over the last dimension, times w if there is one."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(z.clamp(max=30.0))))


# ------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """(f_i, factor on cosine and sine).  f_i = base^(-2i/dims); with ``scaling`` the slow pairs are divided
    by ``factor``: pair number n(t) is the one that turns t times over ``original`` positions, pairs up to
    n(fast) stay, pairs from n(slow) on are slowed, those between are a blend."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F), 1.0
    factor, original = float(sc["factor"]), float(sc["original"])

    def pair(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair(float(sc["fast"]))), 0), min(math.ceil(pair(float(sc["slow"]))), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / factor * r + v * (1.0 - r))
    return torch.tensor(out, dtype=F), 0.1 * math.log(factor) + 1.0


def turn(x, pos, rot, interleaved):
    """x [T, heads, d]: pair i of the first rot.dims dimensions, (2i, 2i + 1) or (i, i + dims/2), (u, v) at
    position p becomes (u c - v s, v c + u s) with c, s = cos, sin of p f_i times the factor."""
    if not rot or not rot["dims"]:
        return x
    f, mag = frequencies(rot)
    out, half = x.clone(), len(f)
    for i in range(half):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + half)
        angle = pos.to(F) * f[i]
        c, s = (torch.cos(angle) * mag)[:, None], (torch.sin(angle) * mag)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a], out[..., b] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------- attention
def sink_softmax_attention(q, k, v, pos_q, pos_k, scale, sink):
    """q [Tq, H, d], k [Tk, H, d], v [Tk, H, dv], sink [H] -> [Tq, H, dv]: weights
    exp(s_j) / (exp(sink_h) + sum_j exp(s_j)) over the keys j <= i."""
    s = torch.einsum("thd,jhd->htj", q, k) * scale
    s = s.masked_fill(~(pos_k[None, :] <= pos_q[:, None])[None], -math.inf)
    z = sink[:, None, None].expand(-1, s.shape[1], 1)
    w = torch.softmax(torch.cat([s, z], -1), -1)[..., :-1]
    return torch.einsum("htj,jhv->thv", w, v)


def latent_attention(h, W, p, m, eps, pos, past, shared):
    """``past``: (latent, rotated key part, positions) of the earlier tokens, or None; ``shared``: the same of
    all tokens so far from the layer named by ``kv_from`` (None: this layer has latents of its own)."""
    T, H, d, r, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms(h @ W[p + "dq"].T, eps, W[p + "dq.norm"]) @ W[p + "uq"].T).view(T, H, d + r)
    q_rot = turn(q[..., d:], pos, m.get("rot"), True)
    if shared is not None:
        c, k_rot, pos_k = shared
    else:
        z = h @ W[p + "dkv"].T
        c, k_rot, pos_k = rms(z[:, :R], eps, W[p + "dkv.norm"]), turn(z[:, None, R:], pos, m.get("rot"), True)[:, 0], pos
        if past is not None:
            c, k_rot, pos_k = torch.cat([past[0], c]), torch.cat([past[1], k_rot]), torch.cat([past[2], pos])
    n = c.shape[0]
    k = torch.cat([(c @ W[p + "uk"].T).view(n, H, d), k_rot[:, None].expand(n, H, r)], -1)
    v = (c @ W[p + "uv"].T).view(n, H, dv)
    o = sink_softmax_attention(torch.cat([q[..., :d], q_rot], -1), k, v, pos, pos_k, m["scale"], W[p + "sink"])
    return o.reshape(T, H * dv) @ W[p + "o"].T, (c, k_rot, pos_k)


def attention(h, W, p, m, eps, pos, past):
    """``past`` = (keys, values, positions): a value is its token's projected key, before norm and rotation."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ W[p + "q"].T + W[p + "q.b"]).view(T, H, d)
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(T, G, d)
    v = k
    q = turn(rms(q, eps, W[p + "q.norm"]), pos, m.get("rot"), False)
    k = turn(rms(k, eps, W[p + "k.norm"]), pos, m.get("rot"), False)
    pos_k = pos
    if past is not None:
        k, v, pos_k = torch.cat([past[0], k]), torch.cat([past[1], v]), torch.cat([past[2], pos])
    kk, vv = k.repeat_interleave(H // G, dim=1), v.repeat_interleave(H // G, dim=1)
    o = sink_softmax_attention(q, kk, vv, pos, pos_k, m["scale"], W[p + "sink"]).reshape(T, H * d)
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T + W[p + "o.b"], (k, v, pos_k)


# ------------------------------------------------------------------------------- delta rule
def short_conv(u, w, before):
    """Causal convolution over time, channel by channel: u [T, C], w [C, taps] (last column: the current
    token), ``before`` [taps - 1, C] the inputs in front of u (zeros before a sequence's start).  Returns
    (y [T, C], the inputs to keep)."""
    taps = w.shape[1]
    full = torch.cat([before, u])
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * full[t + j]
    return y, full[full.shape[0] - (taps - 1):].clone()


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_scan(q, k, v, beta, g, S):
    """S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q, token after token.  q, k [T, H, d],
    v [T, H, dv], beta and g [T, H], S [H, d, dv].  Returns (o [T, H, dv], S)."""
    S, os = S.clone(), []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        os.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(os), S


def delta(h, W, p, m, eps, pos, past):
    """``past`` = (S, the convolutions' last inputs of q, k, v)."""
    T, H, G, d, dv, taps = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], int(m["conv"])
    rows, kept = [], []
    for n, name in enumerate("qkv"):
        u = h @ W[p + name].T
        y, keep = short_conv(u, W[p + name + ".conv"], past[1][n] if past is not None else torch.zeros(taps - 1, u.shape[1], dtype=F))
        rows.append(silu(y))
        kept.append(keep)
    q, k = unit(rows[0].view(T, G, d)) * d ** -0.5, unit(rows[1].view(T, G, d))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ W[p + "b"].T)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    S = past[0] if past is not None else torch.zeros(H, d, dv, dtype=F)
    o, S = delta_scan(q, k, rows[2].view(T, H, dv), beta, g, S)
    o = rms(o, eps, W[p + "norm"]).reshape(T, H * dv) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T, (S, kept)


# ------------------------------------------------------------------------------- feed-forward, model
def feed_forward(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, W, tokens, pos=None, past=None, layer_trace=None):
    """Logits [T, vocab] of ``tokens`` (one sequence) at positions ``pos`` (default 0..T-1) after
    ``past`` (a list with one entry per layer, as returned).  Returns (logits, past)."""
    W = {k: v.to(F) for k, v in W.items()}
    pos = torch.arange(len(tokens)) if pos is None else pos
    eps = float(cfg["norm"]["eps"])
    x = W["embed"][torch.as_tensor(tokens)] * float(cfg["embedding"]["scale"])
    new_past = []
    for i, layer in enumerate(cfg["layers"]):
        p, m, before = f"l{i}.", layer["mixer"], past[i] if past is not None else None
        h = rms(x, eps, W[p + "norm1"])
        if layer["type"] == "latent_attention":
            j = m.get("kv_from")
            y, kept = latent_attention(h, W, p + "mix.", m, eps, pos, before, new_past[j] if j is not None else None)
        elif layer["type"] == "delta":
            y, kept = delta(h, W, p + "mix.", m, eps, pos, before)
        else:
            y, kept = attention(h, W, p + "mix.", m, eps, pos, before)
        new_past.append(kept)
        if layer.get("mlp") is not None:
            y = y + feed_forward(h, W, p + "mlp.")
        x = x + y
        if layer_trace is not None:
            layer_trace.append(x.clone())
    return rms(x, eps, W["final.norm"]) @ W["head"].T, new_past


def tensor_shapes(cfg):
    """name -> shape of every tensor of a model with this configuration."""
    Wd, V = int(cfg["width"]), int(cfg["vocab"])
    out = {"embed": (V, Wd), "head": (V, Wd), "final.norm": (Wd,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.mix.", layer["mixer"]
        H, d = m["heads"], m["dim"]
        out[f"l{i}.norm1"] = (Wd,)
        if layer["type"] == "latent_attention":
            r, dv, R, Q = m["rot_dim"], m["vdim"], m["kv_rank"], m["q_rank"]
            out.update({p + "dq": (Q, Wd), p + "dq.norm": (Q,), p + "uq": (H * (d + r), Q), p + "uk": (H * d, R),
                        p + "uv": (H * dv, R), p + "sink": (H,), p + "o": (Wd, H * dv)})
            if m.get("kv_from") is None:
                out.update({p + "dkv": (R + r, Wd), p + "dkv.norm": (R,)})
        elif layer["type"] == "delta":
            G, dv = m["kv_heads"], m["vdim"]
            for n, c in (("q", G * d), ("k", G * d), ("v", H * dv)):
                out.update({p + n: (c, Wd), p + n + ".conv": (c, int(m["conv"]))})
            out.update({p + "b": (H, Wd), p + "a": (H, Wd), p + "A_log": (H,), p + "dt_bias": (H,), p + "norm": (dv,),
                        p + "g": (H * dv, Wd), p + "o": (Wd, H * dv)})
        else:
            G = m["kv_heads"]
            out.update({p + "q": (H * d, Wd), p + "q.b": (H * d,), p + "k": (G * d, Wd), p + "k.b": (G * d,),
                        p + "q.norm": (d,), p + "k.norm": (d,), p + "sink": (H,), p + "g": (H * d, Wd),
                        p + "o": (Wd, H * d), p + "o.b": (Wd,)})
        if layer.get("mlp") is not None:
            ff = layer["mlp"]["ff"]
            out.update({f"l{i}.mlp.gate": (ff, Wd), f"l{i}.mlp.up": (ff, Wd), f"l{i}.mlp.down": (Wd, ff)})
    return out
