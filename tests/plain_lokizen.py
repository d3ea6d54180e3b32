"""Lokizen, plainly: every mechanism as one slow function in float64, written from the design's equations
and sharing nothing with the engine.  W maps tensor names to torch tensors; tokens is a list of ids.

Notation: x the residual stream [T, width]; N(w, y) = w * y / sqrt(mean(y^2) + eps) over the last axis; U(y) = N(1, y).

    x0 = c embed[token];  x = x0
    per layer run: x <- x + mixer(N(w_1, x));  x <- x + ff(N(w_2, x))        (a looped layer runs several times; ahead of
                                                                              each pass but the first x <- x + x0)
    logits = head N(w_f, x)
"""
import math

import torch

F = torch.float64


def rms_norm(y, w, eps):
    y = y.to(F)
    y = y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)
    return y if w is None else y * w.to(F)


def lin(h, W, name):
    return h.to(F) @ W[name].to(F).T


def bucket(n, rows, farthest):
    """The row of the bias table for distance n.  In floating point, with the logarithm's quotient nudged by an amount
    far below the spacing of its values so that a distance on a bucket's border falls into the farther bucket."""
    half = rows // 2
    if n < half:
        return n
    share = math.log(n / half) / math.log(farthest / half) * (rows - half)
    return min(rows - 1, half + math.floor(share + 1e-9))


def distance_bias(T, table, farthest):
    """[H, T, T]: what each head adds to the score of query i and key j (j <= i)."""
    rows = [bucket(n, table.shape[0], farthest) for n in range(T)]
    by_distance = table.to(F)[torch.tensor(rows)]                       # [T, H]
    d = (torch.arange(T)[:, None] - torch.arange(T)[None, :]).clamp(min=0)
    return by_distance[d].permute(2, 0, 1)


def visible(T, window, keep_first):
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & ((i - j < window) | (j < keep_first)) if window else seen


def softmax_rows(s, mask):
    s = s.masked_fill(~mask, -math.inf)
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def mix_heads(p, talk):
    """w_h = sum_g talk[h, g] p_g for p [H, T, T]."""
    return torch.einsum("hg,gij->hij", talk.to(F), p)


def mixed_attention(q, k, v, scale, table, farthest, talk, window, keep_first):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    k = k.to(F).repeat_interleave(H // G, dim=1)
    v = v.to(F).repeat_interleave(H // G, dim=1)
    s = torch.einsum("ihd,jhd->hij", q.to(F), k) * scale + distance_bias(T, table, farthest)
    return torch.einsum("hij,jhd->ihd", mix_heads(softmax_rows(s, visible(T, window, keep_first)), talk), v)


def attention(h, W, p, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    mask = m.get("mask") or {}
    q = rms_norm(lin(h, W, p + "q"), W[p + "q.norm"], eps).view(T, H, d)       # over all heads at once
    k = rms_norm(lin(h, W, p + "k"), W[p + "k.norm"], eps).view(T, G, d)
    v = lin(h, W, p + "v").view(T, G, dv)
    o = mixed_attention(q, k, v, m["scale"], W[p + "rel"], m["bias_max"], W[p + "talk"], mask.get("size"),
                        mask.get("keep_first", 0))
    return lin(o.reshape(T, H * dv) * torch.sigmoid(lin(h, W, p + "g")), W, p + "o")


def rotate(x, rot):
    """x [T, heads, d]: the first rot.dims elements of every head turned, pair i being (i, i + dims / 2)."""
    if not rot:
        return x
    half = rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(half)], dtype=F)
    a = torch.arange(x.shape[0], dtype=F)[:, None] * f[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def retention_state(q, k, v, decay, S=None):
    """q, k [T, H, d] (rotated, k scaled), v [T, H, dv] -> (read-outs [T, H, dv], S [H, d, dv])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F) if S is None else S
    fade = torch.tensor(decay, dtype=F)[:, None, None]
    out = []
    for t in range(T):
        S = fade * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def silu(z):
    return z * torch.sigmoid(z)


def retention(h, W, p, m, eps):
    T = h.shape[0]
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q = rotate(lin(h, W, p + "q").view(T, H, d), m.get("rot"))
    k = rotate(lin(h, W, p + "k").view(T, H, d), m.get("rot")) * d ** -0.5
    o, _ = retention_state(q, k, lin(h, W, p + "v").view(T, H, dv), m["decay"])
    return lin(rms_norm(o, None, eps).reshape(T, H * dv) * silu(lin(h, W, p + "g")), W, p + "o")


def expert(h, W, p):
    return torch.clamp(lin(h, W, p + "up"), min=0.0) ** 2 @ W[p + "down"].to(F).T


def route(h, W, p, top, scale):
    """-> (chosen experts [T, top], their weights): chosen by logistic score + correction, weighted by the score alone."""
    s = torch.sigmoid(lin(h, W, p + "router"))
    idx = (s + W[p + "correction"].to(F)).topk(top, dim=-1).indices
    return idx, s.gather(-1, idx) * scale


def routed_ff(h, W, p, m):
    idx, w = route(h, W, p, m["router"]["top"], m["router"]["scale"])
    out = torch.zeros(h.shape, dtype=F)
    for e in range(m["router"]["experts"]):
        for c in range(idx.shape[1]):
            hit = idx[:, c] == e
            if bool(hit.any()):
                out[hit] += w[hit, c][:, None] * expert(h[hit], W, p + f"e{e}.")
    return out


def layer_runs(cfg):
    """[(layer, whether the embedding is added first)] in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


MIXERS = {"attention": attention, "retention": retention}


def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out, a list, receives the stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][torch.tensor(tokens)].to(F) * cfg["embedding"]["scale"]
    x = x0
    for i, again in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        if again:
            x = x + x0
        x = x + MIXERS[layer["type"]](rms_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            x = x + routed_ff(rms_norm(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return lin(rms_norm(x, W["final.norm"], eps), W, "head")
