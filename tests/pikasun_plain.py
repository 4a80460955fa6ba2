"""Plain, slow restatement of the Pikasun design in float64 on the CPU: one function per mechanism, whole sequences
at once, no cache, no batching.  TEST INFRASTRUCTURE: it shares no code with the package; the GPU tests compare the
package's kernels, cache and scheduler with it.

Weights are a dict name -> float64 tensor with the checkpoint's names (`embed`, `l<i>.norm1`, `l<i>.norm1.b`,
`l<i>.mix.q`, ..., `final.norm`, `head`); the configuration is the parsed config.json."""
import math

import torch

F64 = torch.float64


# ---- norms -----------------------------------------------------------------------------------------------
def layer_norm(x, weight, bias, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * weight + bias over the last axis."""
    dev = x - x.mean(-1, keepdim=True)
    return dev / torch.sqrt((dev * dev).mean(-1, keepdim=True) + eps) * weight + bias


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


# ---- rotation --------------------------------------------------------------------------------------------
def rotation_frequencies(rot):
    """(angular frequency per rotated pair, magnitude of cos and sin).  With scaling, a linear ramp over the pair index
    slows the pairs that turn fewer than `slow` times within `original` positions by `factor` and keeps those that turn
    more than `fast` times."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return torch.tensor(f, dtype=F64), 1.0
    index_of = lambda turns: dims * math.log(float(sc["original"]) / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo = max(math.floor(index_of(float(sc["fast"]))), 0)
    hi = min(math.ceil(index_of(float(sc["slow"]))), dims - 1)
    out = []
    for i, fi in enumerate(f):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / float(sc["factor"]) * ramp + fi * (1.0 - ramp))
    return torch.tensor(out, dtype=F64), 0.1 * math.log(float(sc["factor"])) + 1.0


def turn(u, v, positions, freq, mag):
    """Pairs (u, v) [T, heads, pairs] turned by their position's angles."""
    ang = torch.tensor(positions, dtype=F64)[:, None] * freq[None, :]
    c, s = (mag * torch.cos(ang))[:, None, :], (mag * torch.sin(ang))[:, None, :]
    return u * c - v * s, v * c + u * s


def rotate_halves(x, positions, rot):
    """x [T, heads, d]: entry i is paired with entry i + dims / 2; what lies past `dims` stays."""
    if not rot:
        return x
    freq, mag = rotation_frequencies(rot)
    n = freq.numel()
    u, v = turn(x[..., :n], x[..., n:2 * n], positions, freq, mag)
    return torch.cat([u, v, x[..., 2 * n:]], dim=-1)


def rotate_neighbours(x, positions, rot):
    """x [T, heads, d]: entry 2 i is paired with entry 2 i + 1; what lies past `dims` stays."""
    if not rot:
        return x
    freq, mag = rotation_frequencies(rot)
    n = freq.numel()
    u, v = turn(x[..., 0:2 * n:2], x[..., 1:2 * n:2], positions, freq, mag)
    return torch.cat([torch.stack([u, v], dim=-1).flatten(-2), x[..., 2 * n:]], dim=-1)


# ---- softmax attention over chosen keys --------------------------------------------------------------------
def attend(q, k, v, scale, first_key):
    """q [T, H, d], k [T, G, d], v [T, G, dv], H a multiple of G; position i sees keys first_key(i) .. i."""
    per = q.shape[1] // k.shape[1]
    k, v = k.repeat_interleave(per, dim=1), v.repeat_interleave(per, dim=1)
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=F64)
    for i in range(q.shape[0]):
        a = first_key(i)
        s = torch.einsum("hd,jhd->hj", q[i], k[a:i + 1]) * scale
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[i] = torch.einsum("hj,jhd->hd", e / e.sum(-1, keepdim=True), v[a:i + 1])
    return out


def chunk_start(i, size):
    """First position of the chunk of `size` positions that holds i (no size: one chunk)."""
    return i // size * size if size > 0 else 0


# ---- mixers ----------------------------------------------------------------------------------------------
def latent_rows(h, w, p, m, eps):
    """What a latent layer caches per token: the normed latent and the rotated key part shared by the heads."""
    R, dr = int(m["kv_rank"]), int(m["rot_dim"])
    y = h @ w[p + "dkv"].T
    c = unit_rms(y[:, :R], eps) * w[p + "dkv.norm"]
    shared = rotate_halves(y[:, R:R + dr].view(-1, 1, dr), list(range(h.shape[0])), m.get("rot"))
    return c, shared


def latent_attention(h, w, p, m, rows):
    """Causal attention whose keys and values are decompressed from `rows`; a sigmoid gate per output entry."""
    T, H, dn, dr, dv = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"])
    c, shared = rows
    q = (h @ w[p + "q"].T).view(T, H, dn + dr)
    q = torch.cat([q[..., :dn], rotate_halves(q[..., dn:], list(range(T)), m.get("rot"))], dim=-1)
    k = torch.cat([(c @ w[p + "uk"].T).view(T, H, dn), shared.expand(T, H, dr)], dim=-1)
    v = (c @ w[p + "uv"].T).view(T, H, dv)
    o = attend(q, k, v, float(m["scale"]), lambda i: 0).reshape(T, H * dv)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def chunked_attention(h, w, p, m, eps):
    """Grouped heads, biased projections, query and key norms over the whole projection, rotation in neighbouring pairs,
    keys of the query's own chunk only, a sigmoid gate per head."""
    T, H, G, dk, dv = h.shape[0], int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = (unit_rms(h @ w[p + "q"].T + w[p + "q.b"], eps) * w[p + "q.norm"]).view(T, H, dk)
    k = (unit_rms(h @ w[p + "k"].T + w[p + "k.b"], eps) * w[p + "k.norm"]).view(T, G, dk)
    v = (h @ w[p + "v"].T + w[p + "v.b"]).view(T, G, dv)
    q, k = (rotate_neighbours(x, list(range(T)), m.get("rot")) for x in (q, k))
    size = int((m.get("mask") or {}).get("size", 0))
    o = attend(q, k, v, float(m["scale"]), lambda i: chunk_start(i, size))
    return (o * sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, H * dv) @ w[p + "o"].T


# ---- feed-forward, output ----------------------------------------------------------------------------------
def capped_ff(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].T, max=limit)
    u = torch.clamp(h @ w[p + "up"].T, min=-limit, max=limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w[p + "down"].T


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def forward(cfg, w, tokens, after_layer=None):
    """Logits [T, vocab] of one whole sequence."""
    eps = float(cfg["norm"]["eps"])
    norm = lambda v, name: layer_norm(v, w[name], w[name + ".b"], eps)
    x, rows = w["embed"][torch.tensor(tokens, dtype=torch.long)], {}
    for i, L in enumerate(cfg["layers"]):
        p, m = f"l{i}.", L["mixer"]
        h = norm(x, p + "norm1")
        if L["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                rows[i] = latent_rows(h, w, p + "mix.", m, eps)
            y = latent_attention(h, w, p + "mix.", m, rows[i if src is None else int(src)])
        elif L["type"] == "attention":
            y = chunked_attention(h, w, p + "mix.", m, eps)
        else:
            raise NotImplementedError(L["type"])
        x = x + y
        if L.get("mlp") is not None:
            x = x + capped_ff(norm(x, p + "norm2"), w, p + "mlp.", float(L["mlp"]["limit"]))
        if after_layer is not None:
            after_layer(i, x)
    z = norm(x, "final.norm") @ w["head"].T * float(cfg["logit_scale"])
    return soft_cap(z, float(cfg["logit_softcap"]))
