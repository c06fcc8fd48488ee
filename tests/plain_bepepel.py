"""Plain, slow Bepepel in float64 on the CPU: the oracle of the tests.  One function per
mechanism, written from the design's equations; nothing here is shared with the package.

Notation: x [T, W] the residual stream, h = N(x) a sublayer's input, p the position of a token in
its sequence (from 0).  Attention: H query heads over G key/value heads, head sizes d (queries and
keys) and dv (values).  Matrix states: S [rows, columns] per head, rows belonging to key channels.
A layer is x <- x + m mixer(N1(x)); x <- x + m ffn(N2(x)) with a layer norm N that has a gain and a bias."""
import math

import torch

F = torch.float64
ROUTING_MARGINS = None  # a list: route() appends (token, gap between the last chosen and the first left-out logit)


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    c = x - x.mean(-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus(z):
    return torch.where(z > 30.0, z, torch.log1p(torch.exp(z.clamp(max=30.0))))


# ------------------------------------------------------------------------------- short convolution
def short_conv(u, w, history):
    """Causal convolution over time, channel by channel: u [T, C], w [C, taps] (last column: the current
    token), history [taps - 1, C] = the values before u (zeros before a sequence's start).  Returns
    (y [T, C], the new history)."""
    taps = w.shape[1]
    full = torch.cat([history, u])
    y = torch.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            y[t] += w[:, j] * full[t + j]
    return y, full[full.shape[0] - (taps - 1):].clone()


# ------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """f_i = base^(-2i/dims); with ``scaling``, by wavelength l = 2 pi / f: shorter than original/high
    stays, longer than original/low is divided by factor, between the two a blend that moves from
    one to the other as original/l goes from low to high."""
    dims, base = int(rot["dims"]), float(rot["base"])
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        sc = rot.get("scaling")
        if sc:
            l = 2 * math.pi / f
            orig, low, high, factor = (float(sc[k]) for k in ("original", "low", "high", "factor"))
            if l > orig / low:
                f = f / factor
            elif l >= orig / high:
                s = (orig / l - low) / (high - low)
                f = (1 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=F)


def turn_pairs(x, pos, freq):
    """x [T, heads, d]: dimensions (2i, 2i + 1) = (u, v) at position p become (u c - v s, v c + u s),
    c, s = cos, sin of p f_i; dimensions from 2 len(freq) on pass."""
    out = x.clone()
    for i, f in enumerate(freq.tolist()):
        a = pos.to(F) * f
        c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ------------------------------------------------------------------------------- attention
def visible(pos_q, pos_k, window, keep_first):
    """[Tq, Tk]: j <= i and (i - j < window, or j < keep_first); window 0: every j <= i."""
    i, j = pos_q.to(torch.int64)[:, None], pos_k.to(torch.int64)[None, :]
    near = (i - j < window) if window else torch.ones(i.shape[0], j.shape[1], dtype=torch.bool)
    return (j <= i) & (near | (j < keep_first))


def softmax_attention(q, k, v, pos_q, pos_k, scale, window, keep_first):
    """q [Tq, H, d], k [Tk, G, d], v [Tk, G, dv] -> [Tq, H, dv]; query head a reads head a // (H / G)."""
    group = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(group, dim=1), v.repeat_interleave(group, dim=1)
    s = torch.einsum("thd,jhd->htj", q, k) * scale
    s = s.masked_fill(~visible(pos_q, pos_k, window, keep_first)[None], -math.inf)
    return torch.einsum("htj,jhv->thv", torch.softmax(s, -1), v)


def attention(h, W, p, m, eps, pos, past=None):
    """``past`` = (k, v, positions, last projected rows of q, k, v)."""
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    taps = int(m["conv"])
    rows, hist = [], []
    for n, name in enumerate("qkv"):
        u = h @ W[p + name].T + W[p + name + ".b"]
        before = past[3][n] if past is not None else torch.zeros(taps - 1, u.shape[1], dtype=F)
        y, kept = short_conv(u, W[p + name + ".conv"], before)
        rows.append(y)
        hist.append(kept)
    q, k, v = rows[0].view(T, H, d), rows[1].view(T, G, d), rows[2].view(T, G, dv)
    if m.get("rot"):
        f = frequencies(m["rot"])
        q, k = turn_pairs(q, pos, f), turn_pairs(k, pos, f)
    q, k = rms(q, eps), rms(k, eps)
    pos_k = pos
    if past is not None:
        k, v, pos_k = torch.cat([past[0], k]), torch.cat([past[1], v]), torch.cat([past[2], pos])
    mask = m.get("mask") or {}
    o = softmax_attention(q, k, v, pos, pos_k, m["scale"], int(mask.get("size") or 0), int(mask.get("keep_first") or 0))
    return o.reshape(T, H * dv) @ W[p + "o"].T, (k, v, pos_k, hist)


# ------------------------------------------------------------------------------- state spaces
def ssd_scan(x, B, C, dt, A_log, D, S):
    """x [T, H, dv], B and C [T, H, N] (each head's own group already picked), dt [T, H] positive:
    S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x.  Returns (y [T, H, dv], S)."""
    S, ys = S.clone(), []
    for t in range(x.shape[0]):
        a = torch.exp(-torch.exp(A_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t][:, :, None] * x[t][:, None, :]
        ys.append(torch.einsum("hnv,hn->hv", S, C[t]) + D[:, None] * x[t])
    return torch.stack(ys), S


def gated_group_norm(y, z, w, groups, eps):
    """y silu(z), divided by the root mean square of its part (``groups`` equal parts), times w."""
    g = y * silu(z)
    return rms(g.view(g.shape[0], groups, -1), eps).reshape(g.shape) * w


def mamba2(h, W, p, m, eps, past=None):
    """``past`` = (S, last inputs of the convolution)."""
    T, H, dv, N, G, taps = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"], int(m["conv"])
    inner = H * dv
    u = h @ W[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    S, before = past if past is not None else (torch.zeros(H, N, dv, dtype=F), torch.zeros(taps - 1, xbc.shape[1], dtype=F))
    y, kept = short_conv(xbc, W[p + "conv"], before)
    xbc = silu(y + W[p + "conv.b"])
    x = xbc[:, :inner].reshape(T, H, dv)
    B, C = (xbc[:, inner + i * G * N:inner + (i + 1) * G * N].reshape(T, G, N).repeat_interleave(H // G, dim=1) for i in (0, 1))
    y, S = ssd_scan(x, B, C, softplus(dt + W[p + "dt_bias"]), W[p + "A_log"], W[p + "D"], S)
    y = gated_group_norm(y.reshape(T, inner), z, W[p + "norm"], m["norm_groups"], eps)
    return y @ W[p + "o"].T, (S, kept)


def parallel(h, W, p, m, eps, pos, past=None):
    left, kept_l = attention(h, W, p + "left.", m["left"], eps, pos, past[0] if past is not None else None)
    right, kept_r = mamba2(h, W, p + "right.", m["right"], eps, past[1] if past is not None else None)
    return m["left_scale"] * left + m["right_scale"] * right, (kept_l, kept_r)


# ------------------------------------------------------------------------------- gated linear attention
def gla_scan(q, k, v, alpha, S):
    """S <- diag(alpha) S + k v^T, o = S^T q; q, k, alpha [T, H, d], v [T, H, dv]."""
    S, os = S.clone(), []
    for t in range(q.shape[0]):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        os.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(os), S


def gla(h, W, p, m, eps, pos, past=None):
    T, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, d) * d ** -0.5
    k, v = (h @ W[p + "k"].T).view(T, H, d), (h @ W[p + "v"].T).view(T, H, dv)
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    alpha = (torch.sigmoid(z) ** (1.0 / m["tau"])).view(T, H, d)
    o, S = gla_scan(q, k, v, alpha, past if past is not None else torch.zeros(H, d, dv, dtype=F))
    o = (rms(o, eps) * W[p + "norm"]).reshape(T, H * dv) * silu(h @ W[p + "g"].T)
    return o @ W[p + "o"].T, S


# ------------------------------------------------------------------------------- feed-forwards
def glu(h, W, p, act):
    return (act(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, r):
    """(experts [T, top], weights [T, top]): the largest logits, weighted by a softmax over those."""
    z = h @ W[p + "router"].T + W[p + "router.b"]
    top, E = int(r["top"]), z.shape[1]
    best = z.topk(min(top + 1, E), dim=-1)
    if ROUTING_MARGINS is not None:
        gap = best.values[:, top - 1] - best.values[:, top] if E > top else torch.full((z.shape[0],), math.inf, dtype=F)
        ROUTING_MARGINS.extend(enumerate(gap.tolist()))
    return best.indices[:, :top], torch.softmax(best.values[:, :top], -1)


def moe(h, W, p, mlp):
    ids, w = route(h, W, p, mlp["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(ids[t].tolist(), w[t]):
            out[t] += a * glu(h[t:t + 1], W, f"{p}e{e}.", silu)[0]
    if mlp.get("shared"):
        out = out + glu(h, W, p + "shared.", silu)
    return out


def feed_forward(h, W, p, mlp):
    return glu(h, W, p, gelu_tanh) if mlp["kind"] == "dense" else moe(h, W, p, mlp)


# ------------------------------------------------------------------------------- the model
MIXERS = {"gla": gla, "parallel": parallel}


def forward(cfg, W, tokens, pos=None, past=None, layer_trace=None):
    """Logits [T, vocab] of ``tokens`` (one sequence) at positions ``pos`` (default 0..T-1) after
    ``past`` (a list with one entry per layer, as returned).  Returns (logits, past)."""
    W = {k: v.to(F) for k, v in W.items()}
    pos = torch.arange(len(tokens)) if pos is None else pos
    eps, mult = float(cfg["norm"]["eps"]), float(cfg["residual_mult"])
    norm = lambda x, name: layer_norm(x, W[name], W[name + ".b"], eps)
    x = W["embed"][torch.as_tensor(tokens)]
    new_past = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y, kept = MIXERS[layer["type"]](norm(x, p + "norm1"), W, p + "mix.", layer["mixer"], eps, pos,
                                        past[i] if past is not None else None)
        new_past.append(kept)
        x = x + mult * y
        if layer.get("mlp") is not None:
            x = x + mult * feed_forward(norm(x, p + "norm2"), W, p + "mlp.", layer["mlp"])
        if layer_trace is not None:
            layer_trace.append(x.clone())
    return norm(x, "final.norm") @ W["head"].T * float(cfg["logit_scale"]), new_past


def tensor_shapes(cfg, rank=16):
    """name -> shape of every tensor of a model with this configuration (``rank``: of the decay maps, or
    a list of them, one per layer; the configuration does not name it)."""
    Wd, V, out = int(cfg["width"]), int(cfg["vocab"]), {}
    out["embed"], out["head"], out["final.norm"], out["final.norm.b"] = (V, Wd), (V, Wd), (Wd,), (Wd,)
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        out[p + "norm1"] = out[p + "norm1.b"] = (Wd,)
        if layer["type"] == "gla":
            H, d, dv = m["heads"], m["dim"], m["vdim"]
            r = rank[i] if isinstance(rank, (list, tuple)) else rank
            out.update({p + "mix.q": (H * d, Wd), p + "mix.k": (H * d, Wd), p + "mix.v": (H * dv, Wd), p + "mix.g": (H * dv, Wd),
                        p + "mix.o": (Wd, H * dv), p + "mix.norm": (dv,), p + "mix.a1": (r, Wd), p + "mix.a2": (H * d, r),
                        p + "mix.a2.b": (H * d,)})
        else:
            a, q = m["left"], p + "mix.left."
            for n, c in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out.update({q + n: (c, Wd), q + n + ".b": (c,), q + n + ".conv": (c, a["conv"])})
            out[q + "o"] = (Wd, a["heads"] * a["vdim"])
            s, q = m["right"], p + "mix.right."
            inner, bc = s["heads"] * s["vdim"], 2 * s["groups"] * s["state"]
            out.update({q + "in": (2 * inner + bc + s["heads"], Wd), q + "conv": (inner + bc, s["conv"]), q + "conv.b": (inner + bc,),
                        q + "dt_bias": (s["heads"],), q + "A_log": (s["heads"],), q + "D": (s["heads"],), q + "norm": (inner,),
                        q + "o": (Wd, inner)})
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        out[p + "norm2"] = out[p + "norm2.b"] = (Wd,)
        unit = lambda q, ff: {q + "gate": (ff, Wd), q + "up": (ff, Wd), q + "down": (Wd, ff)}
        if mlp["kind"] == "dense":
            out.update(unit(p + "mlp.", mlp["ff"]))
        else:
            E = mlp["router"]["experts"]
            for e in range(E):
                out.update(unit(f"{p}mlp.e{e}.", mlp["expert"]["ff"]))
            out.update({p + "mlp.router": (E, Wd), p + "mlp.router.b": (E,)})
            if mlp.get("shared"):
                out.update(unit(p + "mlp.shared.", mlp["shared"]["ff"]))
    return out
