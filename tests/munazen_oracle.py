"""Plain, slow Munazen forward pass for the tests: one function per mechanism, no cache, no kernels, token loops for the
recurrences. Shares no code with the product path. ``cfg`` is the dictionary of a ``config.json``, ``w`` maps tensor names
to tensors; everything runs in the dtype of the weights (float64 by default)."""
import math

import torch


# ---- norms and activations -----------------------------------------------------------------------------------
def unit_rms(x, eps):
    """Last axis divided by its root mean square."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def group_norm(x, weight, groups, eps):
    """Each of ``groups`` consecutive pieces of the last axis divided by its own root mean square, times the gain."""
    size = x.shape[-1] // groups
    parts = [unit_rms(x[..., g * size:(g + 1) * size], eps) for g in range(groups)]
    return torch.cat(parts, -1) * weight


def sigmoid(x):
    return torch.where(x >= 0, 1 / (1 + torch.exp(-x.abs())), torch.exp(-x.abs()) / (1 + torch.exp(-x.abs())))


def log_sigmoid(x):
    return -(torch.log1p(torch.exp(-x.abs())) + (-x).clamp_min(0))


def softplus(x):
    return torch.log1p(torch.exp(-x.abs())) + x.clamp_min(0)


def silu(x):
    return x * sigmoid(x)


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def poly_norm(z, coef, eps):
    """a N(z) + b N(z^2) + c N(z^3) + e; N divides a row by its root mean square."""
    a, b, c, e = coef
    return a * unit_rms(z, eps) + b * unit_rms(z * z, eps) + c * unit_rms(z * z * z, eps) + e


# ---- rotary positions --------------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """(frequencies [dims / 2], factor of cos and sin)."""
    n, sc = rot["dims"], rot.get("scaling")
    plain = [rot["base"] ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return plain, 1.0

    def index_of(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(rot["base"]))
    lo = max(math.floor(index_of(sc["fast"])), 0)
    hi = min(math.ceil(index_of(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        r = min(1.0, max(0.0, (i - lo) / max(hi - lo, 0.001)))
        out.append(f / sc["factor"] * r + f * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def turn_pairs(x, positions, freqs, amp=1.0):
    """x [T, heads, dim]: neighbours 2i and 2i + 1 turn by position * freqs[i]; features behind the last pair pass."""
    out = x.clone()
    for i, f in enumerate(freqs):
        ang = torch.tensor([p * f for p in positions], dtype=torch.float64)
        c, s = (ang.cos() * amp).to(x.dtype)[:, None], (ang.sin() * amp).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def value_frequencies(base, vdim):
    return [base ** (-2.0 * m / vdim) for m in range(vdim // 2)]


# ---- attention with rotated values ---------------------------------------------------------------------------------
def causal_mask(T):
    return torch.tensor([[j <= i for j in range(T)] for i in range(T)])


def masked_softmax_attention(q, k, v, mask, scale):
    """q [T, H, d], k [S, G, d], v [S, G, dv]; mask [T, S]; query head h reads kv head h // (H / G)."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(~mask, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, g]
    return out


def attention(h, m, w, pre):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = list(range(T))
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).reshape(T, H, d)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).reshape(T, G, d)
    v = (h @ w[pre + "v"].T + w[pre + "v.b"]).reshape(T, G, dv)
    freqs, amp = rotary_frequencies(m["rot"])
    vf = value_frequencies(m["rot"]["base"], dv)
    q, k = turn_pairs(q, pos, freqs, amp), turn_pairs(k, pos, freqs, amp)
    o = masked_softmax_attention(q, k, turn_pairs(v, pos, vf), causal_mask(T), m["scale"])
    o = turn_pairs(o, [-p for p in pos], vf)
    o = o * sigmoid(h @ w[pre + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w[pre + "o"].T + w[pre + "o.b"]


# ---- gated linear recurrent unit -----------------------------------------------------------------------------------
def causal_conv(x, weight, bias):
    """x [T, C], weight [C, taps] with the current token's tap last; zeros before the start."""
    T, taps = x.shape[0], weight.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for k in range(taps):
            p = t - (taps - 1) + k
            if p >= 0:
                out[t] = out[t] + weight[:, k] * x[p]
    return out + bias


def block_linear(u, mats, bias):
    """u [T, C] in equal parts, part b through mats[b] ([out, in]) plus bias[b]."""
    size = mats.shape[-1]
    return torch.cat([u[:, b * size:(b + 1) * size] @ mats[b].T + bias[b] for b in range(mats.shape[0])], -1)


def rglru_recurrence(u, r, i, lam, state=None):
    """S_t = a S_(t-1) + sqrt(1 - a^2) i u with log a = -8 r softplus(lam). Returns (S of every token, last S)."""
    S = torch.zeros_like(u[0]) if state is None else state.clone()
    out = torch.empty_like(u)
    for t in range(u.shape[0]):
        log_a = -8 * r[t] * softplus(lam)
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out[t] = S
    return out, S


def rglru(h, w, pre):
    y = gelu_tanh(h @ w[pre + "y"].T + w[pre + "y.b"])
    u = causal_conv(h @ w[pre + "x"].T + w[pre + "x.b"], w[pre + "conv"], w[pre + "conv.b"])
    r = sigmoid(block_linear(u, w[pre + "ra"], w[pre + "ra.b"]))
    i = sigmoid(block_linear(u, w[pre + "ri"], w[pre + "ri.b"]))
    S, _ = rglru_recurrence(u, r, i, w[pre + "lam"])
    return (S * y) @ w[pre + "o"].T


def parallel(h, m, w, pre, eps):
    return m["left_scale"] * attention(h, m["left"], w, pre + "left.") + m["right_scale"] * rglru(h, w, pre + "right.")


# ---- linear attention with a decay per key channel ---------------------------------------------------------------------
def channel_decay_recurrence(q, k, v, log_alpha, state=None):
    """S_t = diag(alpha_t) S_(t-1) + k v^T per head, o = S^T q; q, k, log_alpha [T, H, d], v [T, H, P]."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = torch.exp(log_alpha[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(1)
    return o, S


def gla(h, m, w, pre, eps):
    T, H, d, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[pre + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).reshape(T, H, d)
    v = (h @ w[pre + "v"].T).reshape(T, H, P)
    z = (h @ w[pre + "a1"].T) @ w[pre + "a2"].T + w[pre + "a2.b"]
    o, _ = channel_decay_recurrence(q, k, v, log_sigmoid(z).reshape(T, H, d) / m["tau"])
    o = unit_rms(o, eps) * w[pre + "norm"]
    return (o.reshape(T, H * P) * silu(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- several residual streams --------------------------------------------------------------------------------------
def streams_in(xs, weight):
    """xs [T, streams, D] -> [T, D]."""
    return sum(weight[s] * xs[:, s] for s in range(xs.shape[1]))


def streams_out(xs, y, mix, out):
    """New streams: mix is indexed [from, to], y enters stream t with out[t]."""
    n = xs.shape[1]
    return torch.stack([sum(mix[s, t] * xs[:, s] for s in range(n)) + out[t] * y for t in range(n)], 1)


def layer_runs(cfg):
    """Layer indices in the order they run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    a, b = loop["start"], loop["stop"]
    return list(range(a)) + list(range(a, b)) * loop["times"] + list(range(b, n))


# ---- the model ---------------------------------------------------------------------------------------------------
def forward(tokens, cfg, w, layers_out=None, dtype=torch.float64):
    """tokens: list of ids. Returns logits [T, vocab]; ``layers_out`` (a list) collects the sum of the streams after every
    layer run."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    norm = lambda x, name: group_norm(x, w[name], groups, eps)
    x = w["embed"][torch.as_tensor(tokens)]
    xs = torch.stack([x] * cfg["streams"], 1)
    for i in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        h = norm(streams_in(xs, w[p + "hc1.in"]), p + "norm1")
        y = {"parallel": parallel, "gla": gla}[layer["type"]](h, layer["mixer"], w, p + "mix.", eps)
        xs = streams_out(xs, y, w[p + "hc1.mix"], w[p + "hc1.out"])
        if layer.get("mlp"):
            h = norm(streams_in(xs, w[p + "hc2.in"]), p + "norm2")
            y = poly_norm(h @ w[p + "mlp.up"].T, w[p + "mlp.act"], eps) @ w[p + "mlp.down"].T
            xs = streams_out(xs, y, w[p + "hc2.mix"], w[p + "hc2.out"])
        if layers_out is not None:
            layers_out.append(xs.sum(1))
    return norm(xs.sum(1), "final.norm") @ w["head"].T
