"""Plain, slow Fovudra forward pass for the tests: one function per mechanism, no cache, no kernels, token loops for the
recurrences. Shares no code with the product path. ``cfg`` is the dictionary of a ``config.json``, ``w`` maps tensor names
to tensors; everything runs in the dtype of the weights (float64 by default)."""
import math

import torch


# ---- norms and activations -----------------------------------------------------------------------------------
def unit_rms(x, eps):
    """Last axis divided by its root mean square."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def rms_norm_zero_centred(x, weight, eps):
    return unit_rms(x, eps) * (1 + weight)


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def silu(x):
    return x * sigmoid(x)


def log_sigmoid(x):
    return -(torch.log1p(torch.exp(-x.abs())) + (-x).clamp_min(0))


def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


# ---- rotary positions --------------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """Frequencies [dims / 2]; with scaling, long waves are slowed by the factor and a middle band is blended."""
    n, sc = rot["dims"], rot.get("scaling")
    out = []
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        if sc:
            wave = 2 * math.pi / f
            if wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            elif wave >= sc["original"] / sc["high"]:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: of the first ``dims`` features, i turns together with i + dims / 2."""
    f, half = rotary_frequencies(rot), rot["dims"] // 2
    out = x.clone()
    for t, p in enumerate(positions):
        for i, fi in enumerate(f):
            c, s = math.cos(p * fi), math.sin(p * fi)
            u, v = x[t, ..., i], x[t, ..., i + half]
            out[t, ..., i] = u * c - v * s
            out[t, ..., i + half] = v * c + u * s
    return out


# ---- attention ---------------------------------------------------------------------------------------------------
def visible(i, j, size, keep_first):
    return j <= i and (i - j < size or j < keep_first)


def window_mask(T, size, keep_first):
    m = torch.zeros(T, T, dtype=torch.bool)
    for i in range(T):
        for j in range(T):
            m[i, j] = visible(i, j, size, keep_first)
    return m


def masked_softmax_attention(q, k, v, mask, scale):
    """q [T, H, d], k and v [S, G, d]; mask [T, S]; query head h reads kv head h // (H / G)."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        s = s.masked_fill(~mask, -math.inf)
        e = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (e / e.sum(-1, keepdim=True)) @ v[:, g]
    return out


def attention(h, m, w, pre, eps):
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = list(range(T))
    q = (h @ w[pre + "q"].T + w[pre + "q.b"]).reshape(T, H, d)
    k = (h @ w[pre + "k"].T + w[pre + "k.b"]).reshape(T, G, d)
    v = k
    q = unit_rms(rotate_half(q, pos, m["rot"]), eps)
    k = unit_rms(rotate_half(k, pos, m["rot"]), eps)
    mask = window_mask(T, m["mask"]["size"], m["mask"]["keep_first"])
    o = masked_softmax_attention(q, k, v, mask, m["scale"])
    return o.reshape(T, H * d) @ w[pre + "o"].T


# ---- matrix memories ---------------------------------------------------------------------------------------------
def mlstm_recurrence(q, k, v, i, f, state=None):
    """q, k [T, H, d], v [T, H, P], log gates i, f [T, H]. ``state``: (S [H, d, P], n [H, d], m [H]) or None.
    Returns (o [T, H, P], last state)."""
    T, H, d = q.shape
    P = v.shape[-1]
    if state is None:
        S, n, m = torch.zeros(H, d, P, dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    else:
        S, n, m = (t.clone() for t in state)
    o = torch.empty(T, H, P, dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            top = torch.maximum(f[t, h] + m[h], i[t, h])
            keep, add = torch.exp(f[t, h] + m[h] - top), torch.exp(i[t, h] - top)
            S[h] = keep * S[h] + add * torch.outer(k[t, h], v[t, h])
            n[h] = keep * n[h] + add * k[t, h]
            m[h] = top
            den = torch.maximum((n[h] @ q[t, h]).abs(), torch.exp(-top)) + 1e-6
            o[t, h] = (S[h].T @ q[t, h]) / den
    return o, (S, n, m)


def mlstm(h, m, w, pre, eps):
    T, H, d, P, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = (h @ w[pre + "q"].T).reshape(T, H, d) * d ** -0.5
    k = (h @ w[pre + "k"].T).reshape(T, H, d)
    v = (h @ w[pre + "v"].T).reshape(T, H, P)
    i = soft_cap(h @ w[pre + "i"].T + w[pre + "i.b"], cap)
    f = log_sigmoid(soft_cap(h @ w[pre + "f"].T + w[pre + "f.b"], cap))
    o, _ = mlstm_recurrence(q, k, v, i, f)
    o = unit_rms(o, eps).reshape(T, H * P) * w[pre + "norm"]
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


def decay_recurrence(q, k, v, decay, state=None):
    """S_t = decay S_(t-1) + k v^T per head, o = S^T q. Returns (o [T, H, P], last state [H, d, P])."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    o = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + torch.outer(k[t, h], v[t, h])
            o[t, h] = S[h].T @ q[t, h]
    return o, S


def lightning(h, m, w, pre, eps):
    T, H, d, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w[pre + "q"].T).reshape(T, H, d)
    k = silu(h @ w[pre + "k"].T).reshape(T, H, d)
    v = silu(h @ w[pre + "v"].T).reshape(T, H, P)
    o, _ = decay_recurrence(q, k, v, m["decay"])
    o = unit_rms(o.reshape(T, H * P), eps) * w[pre + "norm"]
    return (o * sigmoid(h @ w[pre + "g"].T)) @ w[pre + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------
def gated_mlp(x, gate, up, down):
    return (silu(x @ gate.T) * (x @ up.T)) @ down.T


def choose_experts(z, top):
    """Per token the ``top`` experts of the largest sigmoid scores and these scores."""
    s = sigmoid(z)
    order = s.argsort(-1, descending=True)[:, :top]
    return order, s.gather(-1, order)


def moe(h, m, w, pre):
    order, weight = choose_experts(h @ w[pre + "router"].T, m["router"]["top"])
    names = lambda e: (w[pre + e + ".gate"], w[pre + e + ".up"], w[pre + e + ".down"])
    out = gated_mlp(h, *names("shared"))
    for t in range(h.shape[0]):
        for e, s in zip(order[t].tolist(), weight[t]):
            out[t] += gated_mlp(s * h[t], *names(f"e{e}"))
    return out


# ---- the model ---------------------------------------------------------------------------------------------------
def forward(tokens, cfg, w, layers_out=None, dtype=torch.float64):
    """tokens: list of ids. Returns logits [T, vocab]; ``layers_out`` (a list) collects the residual after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: rms_norm_zero_centred(x, w[name], eps)
    x = norm(w["embed"][torch.as_tensor(tokens)], "embed.norm")
    mixers = {"attention": attention, "mlstm": mlstm, "lightning": lightning}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm(mixers[layer["type"]](norm(x, p + "norm1"), layer["mixer"], w, p + "mix.", eps), p + "norm1b")
        if layer.get("mlp"):
            x = x + norm(moe(norm(x, p + "norm2"), layer["mlp"], w, p + "mlp."), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T
