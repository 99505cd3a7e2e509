"""Plain, slow Vobunex forward pass for the tests: one function per mechanism, no cache, no kernels, loops where a
loop is the clearest statement. Shares no code with the product path. ``cfg`` is the dictionary of a ``config.json``,
``w`` maps tensor names to tensors; everything runs in the dtype of the weights (float64 by default)."""
import math

import torch


# ---- norms and activations -----------------------------------------------------------------------------------
def layer_norm(x, weight, bias, eps):
    mu = x.mean(-1, keepdim=True)
    var = (x - mu).pow(2).mean(-1, keepdim=True)
    return (x - mu) / (var + eps).sqrt() * weight + bias


def rms_norm(x, weight, eps):
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt() * weight


def grouped_rms_norm(x, weight, parts, eps):
    """Every one of ``parts`` equal pieces of the last axis is divided by its own root mean square."""
    size = x.shape[-1] // parts
    out = torch.empty_like(x)
    for p in range(parts):
        piece = x[..., p * size:(p + 1) * size]
        out[..., p * size:(p + 1) * size] = piece / (piece.pow(2).mean(-1, keepdim=True) + eps).sqrt()
    return out * weight


def silu(x):
    return x / (1 + torch.exp(-x))


# ---- embedding ---------------------------------------------------------------------------------------------------
def embed(tokens, cfg, w):
    x = w["embed"][tokens].clone()
    big = cfg["embedding"].get("bigram")
    if big:
        for t in range(len(tokens)):
            row = big["buckets"] if t == 0 else \
                (int(tokens[t - 1]) * big["mul_prev"] + int(tokens[t]) * big["mul_cur"]) % big["buckets"]
            x[t] += w["bigram"][row]
    return x


# ---- rotary positions --------------------------------------------------------------------------------------------
def rotary_frequencies(rot):
    """(frequencies [dims/2], factor of cos and sin) of one rotary configuration, YaRN-scaled if it says so."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return f, 1.0

    def where(turns):
        return n * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(where(sc["fast"])), 0)
    hi = min(math.ceil(where(sc["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1


def rotate(x, positions, rot):
    """x [T, ..., dims]: neighbours (2i, 2i+1) turn by position * frequency i."""
    f, amp = rotary_frequencies(rot)
    out = x.clone()
    for t, p in enumerate(positions):
        for i, fi in enumerate(f):
            c, s = math.cos(p * fi) * amp, math.sin(p * fi) * amp
            u, v = x[t, ..., 2 * i], x[t, ..., 2 * i + 1]
            out[t, ..., 2 * i] = u * c - v * s
            out[t, ..., 2 * i + 1] = v * c + u * s
    return out


# ---- attention ---------------------------------------------------------------------------------------------------
def sink_softmax(scores, sink):
    """scores [..., n] with -inf where nothing is seen; one extra term exp(sink) in the denominator only."""
    top = torch.maximum(scores.max(-1, keepdim=True).values, sink)
    e = torch.exp(scores - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - top))


def latent_attention(h, m, w, pre, eps):
    T, H, dn, dr, dv, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = list(range(T))
    q = rms_norm(h @ w[pre + "dq"].T, w[pre + "dq.norm"], eps) @ w[pre + "uq"].T
    q = q.reshape(T, H, dn + dr)
    kv = h @ w[pre + "dkv"].T
    c = rms_norm(kv[:, :r], w[pre + "dkv.norm"], eps)
    k_n = (c @ w[pre + "uk"].T).reshape(T, H, dn)
    v = (c @ w[pre + "uv"].T).reshape(T, H, dv)
    q_r = rotate(q[..., dn:], pos, m["rot"])
    k_r = rotate(kv[:, r:], pos, m["rot"])
    out = torch.empty(T, H, dv, dtype=h.dtype)
    mask = torch.ones(T, T, dtype=torch.bool).tril()
    for n in range(H):
        s = (q[:, n, :dn] @ k_n[:, n].T + q_r[:, n] @ k_r.T) * m["scale"]
        s = s.masked_fill(~mask, -math.inf)
        out[:, n] = sink_softmax(s, w[pre + "sink"][n]) @ v[:, n]
    return out.reshape(T, H * dv) @ w[pre + "o"].T


# ---- Mamba-2 -------------------------------------------------------------------------------------------------------
def causal_conv_silu(u, taps, bias):
    """u [T, C], taps [C, K]: the last column weighs the current token, zeros stand before the first."""
    T, K = u.shape[0], taps.shape[1]
    out = torch.empty_like(u)
    for t in range(T):
        acc = bias.clone()
        for k in range(K):
            s = t - (K - 1) + k
            if s >= 0:
                acc = acc + taps[:, k] * u[s]
        out[t] = silu(acc)
    return out


def ssd_recurrence(x, B, C, dt, A_log, D, state=None):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (already positive): token-by-token state update.
    Returns (y [T, H, P], last state [H, N, P])."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = torch.zeros(H, N, P, dtype=x.dtype) if state is None else state.clone()
    y = torch.empty_like(x)
    for t in range(T):
        for n in range(H):
            g = n // (H // G)
            S[n] = torch.exp(-torch.exp(A_log[n]) * dt[t, n]) * S[n] + dt[t, n] * torch.outer(B[t, g], x[t, n])
            y[t, n] = S[n].T @ C[t, g] + D[n] * x[t, n]
    return y, S


def mamba2(h, m, w, pre, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner, gn = H * P, G * N
    z, xbc, dt = (h @ w[pre + "in"].T).split([inner, inner + 2 * gn, H], dim=-1)
    xbc = causal_conv_silu(xbc, w[pre + "conv"], w[pre + "conv.b"])
    x, B, C = xbc.split([inner, gn, gn], dim=-1)
    dt = torch.log1p(torch.exp(-(dt + w[pre + "dt_bias"]).abs())) + (dt + w[pre + "dt_bias"]).clamp_min(0)
    y, _ = ssd_recurrence(x.reshape(T, H, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, w[pre + "A_log"], w[pre + "D"])
    y = grouped_rms_norm(y.reshape(T, inner) * silu(z), w[pre + "norm"], m["norm_groups"], eps)
    return y @ w[pre + "o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------
def relu2_mlp(h, w, pre):
    return (h @ w[pre + "up"].T).clamp_min(0).pow(2) @ w[pre + "down"].T


def clamped_expert(h, gate, up, down, limit):
    g = (h @ gate.T).clamp(max=limit)
    u = (h @ up.T).clamp(-limit, limit)
    return (g / (1 + torch.exp(-1.702 * g)) * (u + 1)) @ down.T


def table_moe(h, tokens, m, w, pre):
    top, limit = m["router"]["top"], m["expert"]["limit"]
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in w[pre + "table"][int(tok)].tolist():
            k = f"{pre}e{e}."
            out[t] += clamped_expert(h[t], w[k + "gate"], w[k + "up"], w[k + "down"], limit) / top
    return out


# ---- the model ---------------------------------------------------------------------------------------------------
def forward(tokens, cfg, w, layers_out=None, dtype=torch.float64):
    """tokens: list of ids. Returns logits [T, vocab]; ``layers_out`` (a list) collects the residual after every layer."""
    w = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in w.items()}
    eps = cfg["norm"]["eps"]
    x = embed(torch.as_tensor(tokens), cfg, w)
    mixers = {"latent_attention": latent_attention, "mamba2": mamba2}
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, w[p + "norm1"], w[p + "norm1.b"], eps)
        x = x + mixers[layer["type"]](h, layer["mixer"], w, p + "mix.", eps)
        mlp = layer.get("mlp")
        if mlp:
            h = layer_norm(x, w[p + "norm2"], w[p + "norm2.b"], eps)
            if mlp["kind"] == "dense":
                x = x + relu2_mlp(h, w, p + "mlp.")
            else:
                x = x + table_moe(h, tokens, mlp, w, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], w["final.norm.b"], eps) @ w["head"].T
