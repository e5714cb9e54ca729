"""Bugidra written plainly: one function per mechanism, whole sequences, no cache, no batching.

A slow restatement of the design's equations for the tests to compare the engine with.  It shares no
code with the engine: weights come as a dict of checkpoint name -> CPU tensor, the configuration as the
dict that config.json holds.  ``dtype`` is the arithmetic's precision (float32 or float64); the
bfloat16 yardstick (``low``) rounds the outputs of projections, short convolutions and activations, and
nothing of what the design computes in 32 bits (angles, scores, softmax, norms, decays, step sizes, unit
vectors and states of the recurrences, the residual sum).

Notation: T tokens at positions t = 0..T-1, width W, H query (or value) heads, G key/value heads, d the size
of a query or key head, e the size of a value head, r the rotated dimensions.
"""
from __future__ import annotations

import math

import torch


def _round(x, low):
    return x if low is None else x.to(low).to(x.dtype)


def linear(x, weight, low=None):
    """y = x W^T, W stored [out, in]; input and result rounded when the arithmetic is low precision."""
    return _round(_round(x, low) @ weight.to(x.dtype).t(), low)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def tanh_norm(x, w, name):
    """Dynamic Tanh: tanh(alpha x) w + b, element by element."""
    return torch.tanh(w[name + ".alpha"].to(x.dtype) * x) * w[name].to(x.dtype) + w[name + ".b"].to(x.dtype)


def silu(x):
    return x * torch.sigmoid(x)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rotary_frequencies(rot):
    """(frequencies f_i of the r / 2 pairs, what cosines and sines are multiplied by), Python floats.

    Unscaled: f_i = base^(-2 i / r), 1.  With ``scaling`` (factor s, original n, fast, slow): a pair that makes more than
    ``fast`` turns over n positions keeps its frequency, one that makes fewer than ``slow`` is slowed by s, with a linear
    ramp between the two pair numbers; cosines and sines grow by 1 + ln(s) / 10."""
    r, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / r) for i in range(r // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0
    pair_of = lambda turns: r * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    first, last = max(math.floor(pair_of(s["fast"])), 0), min(math.ceil(pair_of(s["slow"])), r - 1)
    out = []
    for i, v in enumerate(f):
        ramp = min(max((i - first) / max(last - first, 0.001), 0.0), 1.0)
        out.append(v / s["factor"] * ramp + v * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot, interleaved=False, first=0):
    """x [T, ..., n]: the first r entries are turned in pairs, i with i + r / 2 (or 2 i with 2 i + 1): (u, v) at position
    p becomes (u cos a - v sin a, v cos a + u sin a), a = p f_i.  ``first``: the position of x[0].  Angles are float32
    products of float32 positions and frequencies (float64 when the arithmetic is)."""
    dims = rot["dims"]
    freq, gain = rotary_frequencies(rot)
    kind = torch.float64 if x.dtype == torch.float64 else torch.float32
    f = torch.tensor(freq, dtype=torch.float64).to(kind)
    a = (torch.arange(first, first + x.shape[0], dtype=kind)[:, None] * f[None, :]).to(x.dtype)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = (a.cos() * gain).view(shape), (a.sin() * gain).view(shape)
    pairs = (slice(0, dims, 2), slice(1, dims, 2)) if interleaved else (slice(0, dims // 2), slice(dims // 2, dims))
    u, v = x[..., pairs[0]], x[..., pairs[1]]
    out = x.clone()
    out[..., pairs[0]] = u * cos - v * sin
    out[..., pairs[1]] = v * cos + u * sin
    return out


def causal_attention(q, k, v, scale, cap=None):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e].  Position i sees every j <= i; head a reads key/value head
    floor(a / (H / G)); softmax of (q . k) scale, through cap tanh(. / cap) when there is a cap."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    seen = torch.ones(T, T, dtype=torch.bool).tril()
    for a in range(H):
        g = a // (H // G)
        score = (q[:, a] @ k[:, g].t()) * scale
        if cap:
            score = cap * torch.tanh(score / cap)
        out[:, a] = torch.softmax(score.masked_fill(~seen, float("-inf")), dim=-1) @ v[:, g]
    return out


def unit_attention_mixer(h, w, prefix, m, eps, low=None):
    """The left mixer of a pair: q and k turned by halves, then each head divided by its own root mean square (no
    weight); causal; Wo."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w[prefix + "q"], low).view(T, H, d)
    k = linear(h, w[prefix + "k"], low).view(T, G, d)
    v = linear(h, w[prefix + "v"], low).view(T, G, e)
    q, k = unit_rms(rotate(q, m["rot"]), eps), unit_rms(rotate(k, m["rot"]), eps)
    mixed = _round(causal_attention(_round(q, low), _round(k, low), v, m["scale"]), low)
    return linear(mixed.reshape(T, H * e), w[prefix + "o"], low)


def retention_scan(q, k, v, decay, state=None):
    """q, k [T, H, d], v [T, H, e], decay [H] -> (o [T, H, e], S [H, d, e]): S_t = decay S_(t-1) + k_t v_t^T,
    o_t = S_t^T q_t."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    keep = torch.tensor(decay, dtype=torch.float64).to(q.dtype)[:, None, None]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = keep * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def retention_mixer(h, w, prefix, m, eps, low=None):
    """The right mixer of a pair: q and k turned by halves, k times d^(-1/2); a fixed decay per head; each head's o divided
    by its root mean square; times silu(Wg h); Wo."""
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = rotate(linear(h, w[prefix + "q"], low).view(T, H, d), m["rot"])
    k = rotate(linear(h, w[prefix + "k"], low).view(T, H, d), m["rot"]) * d ** -0.5
    v = linear(h, w[prefix + "v"], low).view(T, H, e)
    o, _ = retention_scan(q, k, v, m["decay"])
    mixed = _round(unit_rms(o, eps).reshape(T, H * e) * silu(linear(h, w[prefix + "g"], low)), low)
    return linear(mixed, w[prefix + "o"], low)


def parallel_mixer(h, w, prefix, m, eps, low=None):
    """Half the sum of the two mixers' outputs, each divided by its root mean square over the width, times a weight."""
    left = unit_attention_mixer(h, w, prefix + "left.", m["left"], eps, low)
    right = retention_mixer(h, w, prefix + "right.", m["right"], eps, low)
    return 0.5 * (unit_rms(left, eps) * w[prefix + "left.out"].to(h.dtype)
                  + unit_rms(right, eps) * w[prefix + "right.out"].to(h.dtype))


def mixed_values(v, first, share):
    """(1 - share) v + share first, ``share`` a learned number."""
    share = share.to(v.dtype)
    return (1.0 - share) * v + share * first


def gated_attention_mixer(h, w, prefix, m, eps, low=None, first_values=None):
    """Grouped attention: q and k divided by the root mean square of the whole projection, times a weight per element;
    turned by neighbours; capped scores; values mixed with the first value-mixing layer's of the same token
    (``first_values``: a list that holds them once there are any); the heads' outputs times sigmoid(Wg h); Wo."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(linear(h, w[prefix + "q"], low), eps) * w[prefix + "q.norm"].to(h.dtype)
    k = unit_rms(linear(h, w[prefix + "k"], low), eps) * w[prefix + "k.norm"].to(h.dtype)
    q, k = rotate(q.view(T, H, d), m["rot"], True), rotate(k.view(T, G, d), m["rot"], True)
    v = linear(h, w[prefix + "v"], low)
    if m.get("v_mix"):
        if first_values:
            v = _round(mixed_values(v, first_values[0], w[prefix + "vmix"]), low)
        else:
            first_values.append(v)
    mixed = causal_attention(_round(q, low), _round(k, low), v.view(T, G, e), m["scale"], m.get("softcap"))
    mixed = _round(mixed.reshape(T, H * e), low)
    mixed = _round(mixed * torch.sigmoid(linear(h, w[prefix + "g"], low)), low)
    return linear(mixed, w[prefix + "o"], low)


def short_conv(u, taps, history=None):
    """y_t[c] = sum_j taps[c, j] u_(t - n + 1 + j)[c] for n taps, zeros (or ``history`` [n - 1, channels]) before u[0]."""
    n = taps.shape[1]
    before = torch.zeros(n - 1, u.shape[1], dtype=u.dtype) if history is None else history
    padded = torch.cat([before, u])
    return sum(padded[j:j + u.shape[0]] * taps[:, j].to(u.dtype) for j in range(n))


def unit_vector(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last dimension."""
    return x / torch.sqrt(x.pow(2).sum(dim=-1, keepdim=True) + 1e-6)


def delta_decay(a, a_log, dt_bias):
    """exp(-exp(A_log) softplus(a + dt)), one per head."""
    return torch.exp(-torch.exp(a_log.to(a.dtype)) * torch.nn.functional.softplus(a + dt_bias.to(a.dtype), threshold=1e9))


def delta_scan(q, k, v, g, beta, state=None):
    """q, k [T, H, d], v [T, H, e], g, beta [T, H] -> (o [T, H, e], S [H, d, e]), per head and in this order
    S <- g S,  u = beta (v - S^T k),  S <- S + k u^T,  o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(dim=1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def delta_mixer(h, w, prefix, m, eps, low=None):
    """The gated delta rule: q, k, v through a short convolution and silu, q and k unit vectors per head, q times
    d^(-1/2); each head's o divided by its root mean square, times a weight of e and silu(Wg h); Wo."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def convolved(name):
        y = _round(short_conv(linear(h, w[prefix + name], low), w[prefix + name + ".conv"]), low)
        return _round(silu(y), low)

    spread = lambda x: x.repeat_interleave(H // G, dim=1)
    q = spread(unit_vector(convolved("q").view(T, G, d)) * d ** -0.5)
    k = spread(unit_vector(convolved("k").view(T, G, d)))
    v = convolved("v").view(T, H, e)
    beta = torch.sigmoid(linear(h, w[prefix + "b"], low))
    g = delta_decay(linear(h, w[prefix + "a"], low), w[prefix + "A_log"], w[prefix + "dt_bias"])
    o, _ = delta_scan(q, k, v, g, beta)
    mixed = unit_rms(o, eps) * w[prefix + "norm"].to(o.dtype)
    mixed = _round(mixed.reshape(T, H * e) * silu(linear(h, w[prefix + "g"], low)), low)
    return linear(mixed, w[prefix + "o"], low)


def feed_forward(h, w, prefix, low=None):
    """down(gelu_tanh(gate h) * (up h))."""
    inner = _round(gelu_tanh(linear(h, w[prefix + "gate"], low)) * linear(h, w[prefix + "up"], low), low)
    return linear(inner, w[prefix + "down"], low)


MIXERS = {"parallel": parallel_mixer, "attention": gated_attention_mixer, "delta": delta_mixer}


def forward(config, w, tokens, dtype=torch.float64, low=None, return_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = w["embed"][tokens].to(dtype) * (config.get("embedding") or {}).get("scale", 1.0)
    after, first_values = [], []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = _round(tanh_norm(x, w, p + "norm1"), low)
        more = (first_values,) if layer["type"] == "attention" else ()
        x = x + MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, low, *more)
        if layer.get("mlp") is not None:
            x = x + feed_forward(_round(tanh_norm(x, w, p + "norm2"), low), w, p + "mlp.", low)
        after.append(x.clone())
    logits = _round(tanh_norm(x, w, "final.norm"), low) @ w["head"].to(dtype).t()
    return (logits, torch.stack(after)) if return_layers else logits
