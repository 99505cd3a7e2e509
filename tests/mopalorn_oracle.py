"""Plain, slow Mopalorn in fp64: one function per mechanism, one sequence, no cache. ``cfg`` is the dictionary of a config.json, ``w``
maps checkpoint names to tensors. Nothing here is shared with the package."""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def turn_halves(x, base, pos=None):
    """x (T, ..., d): features i and i + d / 2 turn together by position * base^(-2 i / d); positions 0, 1, .. or ``pos``."""
    T, d = x.shape[0], x.shape[-1]
    pos = torch.arange(T) if pos is None else torch.tensor(pos)
    out = x.clone()
    for i in range(d // 2):
        a = pos.double() * base ** (-2.0 * i / d)
        a = a.reshape([T] + [1] * (x.dim() - 2))
        u, v = x[..., i], x[..., i + d // 2]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + d // 2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def query_factor(pos, coef, every):
    return 1.0 + coef * math.log((pos + 1) // every + 1)


def cap(s, c):
    return c * torch.tanh(s / c)


def xielu(z, p, q):
    sp = lambda t: math.log1p(math.exp(t))
    neg = z.clamp_max(0)
    return torch.where(z > 0, sp(p) * z * z + z / 2, (0.5 + sp(q)) * (torch.exp(neg) - 1 - neg) + z / 2)


def seen_tokens(T, size=None):
    """(T, T): which keys a query sees."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) if size is None else (j <= i) & (i - j < size)


def block_means(x, P):
    """Means over the whole blocks of P rows of x (T, ...)."""
    n = x.shape[0] // P
    return torch.stack([x[b * P:(b + 1) * P].mean(0) for b in range(n)]) if n else x[:0]


def seen_blocks(T, P, size):
    """(T, T // P): a block is seen once its last token has left the window."""
    i, b = torch.arange(T)[:, None], torch.arange(T // P)[None, :]
    return b * P + P - 1 <= i - size


def weights_of(scores, seen, sink=None):
    """Softmax over the seen keys (last axis); ``sink`` joins the denominator."""
    s = scores.masked_fill(~seen, -math.inf)
    m = s.max(-1, keepdim=True).values
    if sink is not None:
        m = torch.maximum(m, sink)
    e = torch.exp(s - m)
    d = e.sum(-1, keepdim=True)
    if sink is not None:
        d = d + torch.exp(sink - m)
    return e / d


def mixed_values(v, first, lam):
    return (1 - lam) * v + lam * first


def latent_attention(h, m, w, p, eps):
    T, H, dn, dr, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w[p + "q"].T).reshape(T, H, dn + dr)
    ckr = h @ w[p + "dkv"].T
    c = rms(ckr[:, :R], eps) * w[p + "dkv.norm"]
    base = m["rot"]["base"]
    qr, kr = turn_halves(q[..., dn:], base), turn_halves(ckr[:, R:], base)
    k = (c @ w[p + "uk"].T).reshape(T, H, dn)
    v = (c @ w[p + "uv"].T).reshape(T, H, dv)
    s = (torch.einsum("ihd,jhd->hij", q[..., :dn], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    a = weights_of(s, seen_tokens(T, m["mask"]["size"]))
    o = torch.einsum("hij,jhd->ihd", a, v).reshape(T, H * dv)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def heads_of(h, m, w, p, first):
    """q (T, H, d), k, v (T, H, d) repeated over the query heads of their kv head, and the projected values (T, G, dv)."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = (h @ w[p + "k"].T).reshape(T, G, m["dim"])
    raw = (h @ w[p + "v"].T).reshape(T, G, m["vdim"])
    v = raw
    if m.get("v_mix") and first is not None:
        v = mixed_values(raw, first.reshape(raw.shape), w[p + "vmix"])
    of = torch.arange(H) // (H // G)
    return q, k[:, of], v[:, of], raw


def attention(h, m, w, p, first):
    T = h.shape[0]
    q, k, v, raw = heads_of(h, m, w, p, first)
    t = m["q_temp"]
    q = q * torch.tensor([query_factor(i, t["coef"], t["every"]) for i in range(T)], dtype=q.dtype)[:, None, None]
    s = cap(torch.einsum("ihd,jhd->hij", q, k) * m["scale"], m["softcap"])
    o = torch.einsum("hij,jhd->ihd", weights_of(s, seen_tokens(T)), v)
    return o.reshape(T, -1) @ w[p + "o"].T, raw


def attention_2(h, m, w, p, first):
    T = h.shape[0]
    q, k, v, raw = heads_of(h, m, w, p, first)
    P, size = m["mask"]["pool"], m["mask"]["size"]
    kk, vv = torch.cat([k, block_means(k, P)]), torch.cat([v, block_means(v, P)])
    s = torch.einsum("ihd,jhd->hij", q, kk) * m["scale"]
    seen = torch.cat([seen_tokens(T, size), seen_blocks(T, P, size)], 1)
    o = torch.einsum("hij,jhd->ihd", weights_of(s, seen, w[p + "sink"][:, None, None]), vv)
    return o.reshape(T, -1) @ w[p + "o"].T, raw


def feed_forward(h, w, p):
    a, b = (float(t) for t in w[p + "act"])
    return xielu(h @ w[p + "up"].T, a, b) @ w[p + "down"].T


def forward(tokens, cfg, weights, layers=None):
    """Logits (T, V) fp64 of one sequence; ``layers`` collects the residual after every layer."""
    w = {k: t.double().cpu() for k, t in weights.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: rms(x, eps) * w[name]
    x = w["embed"][torch.tensor(tokens)]
    first = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "latent_attention":
            y = latent_attention(h, m, w, p + "mix.", eps)
        else:
            y, raw = {"attention": attention, "attention_2": attention_2}[layer["type"]](h, m, w, p + "mix.", first)
            if m.get("v_mix") and first is None:
                first = raw
        x = x + norm(y, p + "norm1b")
        if layer["mlp"]:
            x = x + norm(feed_forward(norm(x, p + "norm2"), w, p + "mlp."), p + "norm2b")
        if layers is not None:
            layers.append(x)
    return norm(x, "final.norm") @ w["embed"].T * cfg["logit_scale"]
