"""Mapovik, plainly: every mechanism as one slow function in float64, written from the design's equations and
sharing nothing with the engine.  W maps tensor names to torch tensors; tokens is a list of ids.

Notation: x the residual stream [T, width]; L(w, y) = w (y - mean) / sqrt(mean((y - mean)^2) + eps) over the last axis;
N(w, y) = w y / sqrt(mean(y^2) + eps).

    x0 = embed[token];  x = x0
    ahead of pass t of the looped layers (t = 0, 1, ...):  x <- W_in [x; x0] + step_t
    per layer run:  x <- x + m mixer(L(w_1, x));  x <- x + m ff(L(w_2, x))
    logits = c head L(w_f, x)
"""
import torch

F = torch.float64


def layer_norm(y, w, eps):
    y = y.to(F)
    d = y - y.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w.to(F)


def rms_norm(y, w, eps):
    y = y.to(F)
    y = y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w.to(F)


def lin(h, W, name):
    return h.to(F) @ W[name].to(F).T


def silu(z):
    return z / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def conv(u, w, b=None, before=None):
    """u [T, C], w [C, taps] (the last column weighs the current token); before [taps - 1, C]: what came ahead (zeros)."""
    taps = w.shape[1]
    u = u.to(F)
    before = torch.zeros(taps - 1, u.shape[1], dtype=F) if before is None else before.to(F)
    padded = torch.cat([before, u])
    y = sum(padded[j:j + u.shape[0]] * w[:, j].to(F) for j in range(taps))
    return y if b is None else y + b.to(F)


def rotate(x, rot):
    """x [T, heads, d]: pair (i, i + dims / 2) of the first rot.dims elements of every head turned by p f_i, the
    frequencies f_i = base^(-2 i / dims) divided by scaling.factor."""
    if not rot:
        return x
    half = rot["dims"] // 2
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    f = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) / factor for i in range(half)], dtype=F)
    a = torch.arange(x.shape[0], dtype=F)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def attend(q, k, v, scale):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]: causal softmax."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k = k.to(F).repeat_interleave(H // G, dim=1)
    v = v.to(F).repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q.to(F), k) * scale
    s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -float("inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return torch.einsum("hij,jhd->ihd", e / e.sum(-1, keepdim=True), v)


def attention(h, W, p, m):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(lin(h, W, p + "q").view(T, H, d), m.get("rot"))
    k = rotate(lin(h, W, p + "k").view(T, G, d), m.get("rot"))
    o = attend(q, k, lin(h, W, p + "v").view(T, G, dv), m["scale"])
    return lin(o.reshape(T, H * dv), W, p + "o")


def scalar_decay_state(x, B, C, dt, A_log, S=None):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (behind its softplus), A_log [H] -> (read-outs [T, H, P], S [H, N, P]):
    S <- exp(-exp(A_log) dt) S + dt B x^T;  y = S^T C."""
    T, H, P = x.shape
    rep = H // B.shape[1]
    B, C = B.to(F).repeat_interleave(rep, dim=1), C.to(F).repeat_interleave(rep, dim=1)
    S = torch.zeros(H, B.shape[-1], P, dtype=F) if S is None else S
    keep = torch.exp(-torch.exp(A_log.to(F)) * dt.to(F))
    out = []
    for t in range(T):
        S = keep[t][:, None, None] * S + dt[t].to(F)[:, None, None] * B[t][:, :, None] * x[t].to(F)[:, None, :]
        out.append(torch.einsum("hnp,hn->hp", S, C[t]))
    return torch.stack(out), S


def grouped_norm(y, w, groups, eps):
    T, n = y.shape
    return rms_norm(y.view(T, groups, n // groups), None, eps).reshape(T, n) * w.to(F)


def state_space(h, W, p, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    u = lin(h, W, p + "in")
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
    xbc = silu(conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x = xbc[:, :inner].view(T, H, P)
    B = xbc[:, inner:inner + G * N].view(T, G, N)
    C = xbc[:, inner + G * N:].view(T, G, N)
    dt = softplus(dt + W[p + "dt_bias"].to(F))
    y, _ = scalar_decay_state(x, B, C, dt, W[p + "A_log"])
    y = (y + W[p + "D"].to(F)[:, None] * x).reshape(T, inner) * silu(z)
    return lin(grouped_norm(y, W[p + "norm"], m["norm_groups"], eps), W, p + "o")


def parallel(h, W, p, m, eps):
    left = attention(h, W, p + "left.", m["left"])
    right = state_space(h, W, p + "right.", m["right"], eps)
    return 0.5 * (rms_norm(left, W[p + "left.out"], eps) + rms_norm(right, W[p + "right.out"], eps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def channel_delta_state(q, k, v, beta, g, S=None):
    """q, k [T, G, d] (unit vectors, q scaled), v [T, H, dv], beta [T, H], g [T, H, d] -> (read-outs [T, H, dv], S [H, d, dv]):
    S <- diag(g) S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q."""
    T, H = beta.shape
    rep = H // q.shape[1]
    q, k = q.to(F).repeat_interleave(rep, dim=1), k.to(F).repeat_interleave(rep, dim=1)
    S = torch.zeros(H, q.shape[-1], v.shape[-1], dtype=F) if S is None else S
    out = []
    for t in range(T):
        S = g[t].to(F)[:, :, None] * S
        u = beta[t].to(F)[:, None] * (v[t].to(F) - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def channel_decay(a, dt_bias, A_log, H):
    """a [T, H d] (the low-rank projection), dt_bias [H d], A_log [H] -> g [T, H, d]."""
    T = a.shape[0]
    rate = softplus(a.to(F) + dt_bias.to(F)).view(T, H, -1)
    return torch.exp(-torch.exp(A_log.to(F))[:, None] * rate)


def channel_delta(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(conv(lin(h, W, p + n), W[p + n + ".conv"])) for n in "qkv")
    q = unit(q.view(T, G, d)) * d ** -0.5
    k = unit(k.view(T, G, d))
    beta = torch.sigmoid(lin(h, W, p + "b"))
    g = channel_decay(lin(lin(h, W, p + "a1"), W, p + "a2"), W[p + "dt_bias"], W[p + "A_log"], H)
    o, _ = channel_delta_state(q, k, v.view(T, H, dv), beta, g)
    gate = torch.sigmoid(lin(lin(h, W, p + "g1"), W, p + "g2")).view(T, H, dv)
    return lin((rms_norm(o, W[p + "norm"], eps) * gate).reshape(T, H * dv), W, p + "o")


def dense_ff(h, W, p):
    return torch.clamp(lin(h, W, p + "up"), min=0.0) ** 2 @ W[p + "down"].to(F).T


def expert(h, W, p):
    return lin(silu(lin(h, W, p + "gate")) * lin(h, W, p + "up"), W, p + "down")


def table_ff(h, W, p, m, tokens):
    """The experts of a token are a row of a table by its id, each with the weight 1 / top."""
    rows = W[p + "table"].long()[torch.tensor(tokens)]                   # [T, top]
    out = torch.zeros(h.shape, dtype=F)
    for e in range(m["router"]["experts"]):
        for c in range(rows.shape[1]):
            hit = rows[:, c] == e
            if bool(hit.any()):
                out[hit] += expert(h[hit], W, p + f"e{e}.") / m["router"]["top"]
    return out


def layer_runs(cfg):
    """[(layer, the pass that begins ahead of it or None)] in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    runs = [(i, None) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, None) for i in range(loop["stop"], n)]


MIXERS = {"parallel": parallel, "channel_delta": channel_delta}


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out, a list, receives the stream after every layer run."""
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x0 = W["embed"][torch.tensor(tokens)].to(F)
    x = x0
    for i, begins in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if begins is not None:
            x = lin(torch.cat([x, x0], dim=-1), W, "loop.in") + W["loop.step"][begins].to(F)
        x = x + m * MIXERS[layer["type"]](layer_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            h = layer_norm(x, W[p + "norm2"], eps)
            x = x + m * (table_ff(h, W, p + "mlp.", layer["mlp"], tokens) if layer["mlp"]["kind"] == "moe"
                         else dense_ff(h, W, p + "mlp."))
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(layer_norm(x, W["final.norm"], eps), W, "head") * cfg["logit_scale"]
