"""Lotazen written plainly: one function per mechanism, whole sequences, no cache, no batching.

A slow restatement of the design's equations for the tests to compare the engine with.  It shares no
code with the engine: weights come as a dict of checkpoint name -> CPU tensor, the configuration as the
dict that config.json holds.  ``dtype`` is the arithmetic's precision (float32 or float64); the
bfloat16 yardstick (``low``) rounds the outputs of projections and activations, and nothing of what the
design computes in 32 bits (angles, scores, softmax, norms, routers, gates and states of the recurrences,
the residual sum).

Notation: T tokens at positions t = 0..T-1, width W, H query heads, G key/value heads, d the size of a
query or key head, e the size of a value head, r the rotated dimensions, n the size of a window, E experts
of which a token uses K.
"""
from __future__ import annotations

import torch


def _round(x, low):
    return x if low is None else x.to(low).to(x.dtype)


def linear(x, weight, low=None):
    """y = x W^T, W stored [out, in]; input and result rounded when the arithmetic is low precision."""
    return _round(_round(x, low) @ weight.to(x.dtype).t(), low)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last dimension."""
    return x / torch.sqrt(x.pow(2).mean(dim=-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    """The root-mean-square norm with one number for all coordinates."""
    return unit_rms(x, eps) * gain.to(x.dtype)


def rotate_neighbours(x, rot, first=0):
    """x [T, ..., n]: of the first r entries, 2 i pairs with 2 i + 1; the pair (u, v) at position p becomes
    (u cos a - v sin a, v cos a + u sin a), a = p f_i, f_i = base^(-2 i / r) / factor.  ``first``: the position of
    x[0].  Angles are float32 products of float32 positions and frequencies (float64 when the arithmetic is)."""
    dims = rot["dims"]
    factor = (rot.get("scaling") or {}).get("factor", 1.0)
    kind = torch.float64 if x.dtype == torch.float64 else torch.float32
    f = torch.tensor([rot["base"] ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=torch.float64).to(kind)
    a = (torch.arange(first, first + x.shape[0], dtype=kind)[:, None] * f[None, :]).to(x.dtype)
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [dims // 2]
    cos, sin = a.cos().view(shape), a.sin().view(shape)
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def window_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e].  Position i sees j with 0 <= i - j < n; head a reads
    key/value head floor(a / (H / G)); softmax of (q . k) scale."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for i in range(T):
        first = max(0, i - window + 1)
        for a in range(H):
            g = a // (H // G)
            p = torch.softmax((k[first:i + 1, g] @ q[i, a]) * scale, dim=0)
            out[i, a] = p @ v[first:i + 1, g]
    return out


def window_attention_mixer(h, w, prefix, m, eps, low=None):
    """Grouped attention: q, k turned by neighbours on their first r dimensions and then each head divided by its own
    root mean square (no weight); a sliding window; Wo."""
    T = h.shape[0]
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = linear(h, w[prefix + "q"], low).view(T, H, d)
    k = linear(h, w[prefix + "k"], low).view(T, G, d)
    v = linear(h, w[prefix + "v"], low).view(T, G, e)
    q = unit_rms(rotate_neighbours(q, m["rot"]), eps)
    k = unit_rms(rotate_neighbours(k, m["rot"]), eps)
    mixed = _round(window_attention(_round(q, low), _round(k, low), v, m["scale"], m["mask"]["size"]), low)
    return linear(mixed.reshape(T, H * e), w[prefix + "o"], low)


def forget_gate(z, bias, lower):
    """f = l + (1 - l) sigmoid(z + b), channel by channel."""
    lower = lower.to(z.dtype)
    return lower + (1.0 - lower) * torch.sigmoid(z + bias.to(z.dtype))


def tied_gate_scan(q, f, v, state=None):
    """q, f [T, H, d], v [T, H, e] -> (o [T, H, e], S [H, d, e]): S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,
    o_t = S_t^T q_t."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for t in range(T):
        S = f[t][:, :, None] * S + (1.0 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(dim=1)
    return out, S


def hgrn2_mixer(h, w, prefix, m, eps, low=None):
    """Linear attention whose forget gate also decides what is written: q = silu(Wq h), v = Wv h,
    f = l + (1 - l) sigmoid(Wf h + b); each head's o normed over its e values (one weight of e); Wo."""
    T = h.shape[0]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    q = linear(h, w[prefix + "q"], low)
    q = _round(q * torch.sigmoid(q), low).view(T, H, d)
    f = forget_gate(linear(h, w[prefix + "f"], low), w[prefix + "f.b"], w[prefix + "lower"]).view(T, H, d)
    v = linear(h, w[prefix + "v"], low).view(T, H, e)
    o, _ = tied_gate_scan(q, f, v)
    mixed = _round(unit_rms(o, eps) * w[prefix + "norm"].to(o.dtype), low)
    return linear(mixed.reshape(T, H * e), w[prefix + "o"], low)


def parallel_mixer(h, w, prefix, m, eps, low=None):
    """left_scale * window attention + right_scale * HGRN2, both of the same h."""
    left = window_attention_mixer(h, w, prefix + "left.", m["left"], eps, low)
    right = hgrn2_mixer(h, w, prefix + "right.", m["right"], eps, low)
    return m["left_scale"] * left + m["right_scale"] * right


def capped(z, cap):
    return cap * torch.tanh(z / cap)


def mlstm_scan(q, k, v, log_i, log_f, state=None):
    """q, k [T, H, d], v [T, H, e], log_i, log_f [T, H] -> (o [T, H, e], (S, n, m)).

        m_t = max(f_t + m_(t-1), i_t)                   m starts at 0
        S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t the same with k_t alone
        o_t = S_t^T q_t / (max(|n_t . q_t|, exp(-m_t)) + 1e-6)
    """
    T, H, d = q.shape
    e = v.shape[-1]
    if state is None:
        state = torch.zeros(H, d, e, dtype=q.dtype), torch.zeros(H, d, dtype=q.dtype), torch.zeros(H, dtype=q.dtype)
    S, n, m = state
    out = torch.zeros(T, H, e, dtype=q.dtype)
    for t in range(T):
        m_next = torch.maximum(log_f[t] + m, log_i[t])
        keep, write = torch.exp(log_f[t] + m - m_next), torch.exp(log_i[t] - m_next)
        m = m_next
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        size = torch.maximum((n * q[t]).sum(dim=-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(dim=1) / size[:, None]
    return out, (S, n, m)


def mlstm_mixer(h, w, prefix, m, eps, low=None):
    """Matrix memory: q = Wq h d^(-1/2), k = Wk h, v = Wv h; log gates per head, capped by cap tanh(. / cap), the forget
    gate through a log sigmoid; each head's o divided by its own root mean square, all heads times ``norm`` and
    sigmoid(Wg h); Wo."""
    T = h.shape[0]
    H, d, e, cap = m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = linear(h, w[prefix + "q"], low).view(T, H, d) * d ** -0.5
    k = linear(h, w[prefix + "k"], low).view(T, H, d)
    v = linear(h, w[prefix + "v"], low).view(T, H, e)
    log_i = capped(linear(h, w[prefix + "i"], low) + w[prefix + "i.b"].to(h.dtype), cap)
    log_f = torch.nn.functional.logsigmoid(capped(linear(h, w[prefix + "f"], low) + w[prefix + "f.b"].to(h.dtype), cap))
    o, _ = mlstm_scan(q, k, v, log_i, log_f)
    mixed = unit_rms(o, eps).reshape(T, H * e) * w[prefix + "norm"].to(o.dtype)
    mixed = _round(mixed * torch.sigmoid(linear(h, w[prefix + "g"], low)), low)
    return linear(mixed, w[prefix + "o"], low)


SWISH_ALPHA = 1.702


def clamped_expert(x, w, prefix, limit, low=None):
    """g = min(gate x, L), u = clamp(up x, -L, L); down(g sigmoid(1.702 g) (u + 1))."""
    g = torch.clamp(linear(x, w[prefix + "gate"], low), max=limit)
    u = torch.clamp(linear(x, w[prefix + "up"], low), min=-limit, max=limit)
    return linear(_round(g * torch.sigmoid(SWISH_ALPHA * g) * (u + 1.0), low), w[prefix + "down"], low)


def route(h, router, top, low=None):
    """Scores = sigmoid(R h); the ``top`` largest are chosen (the lower index wins a tie) and are the weights as they
    are.  Returns (chosen [T, K], weights [T, K])."""
    scores = torch.sigmoid(_round(h, low) @ router.to(h.dtype).t())
    order = torch.sort(scores, dim=-1, descending=True, stable=True).indices[:, :top]
    return order, torch.gather(scores, 1, order)


def routed_experts(h, w, prefix, mlp, low=None, margins=None):
    """sum over a token's chosen experts of expert_e(score_e h), plus the shared expert of h.  ``margins``: a list
    that receives, per token, by how much the last chosen output of the router leads the first rejected one."""
    top = mlp["router"]["top"]
    chosen, weights = route(h, w[prefix + "router"], top, low)
    if margins is not None and top < mlp["router"]["experts"]:
        ranked = (h @ w[prefix + "router"].to(h.dtype).t()).sort(dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for n in range(top):
            row = weights[t, n] * _round(h[t:t + 1], low)
            out[t] += clamped_expert(row, w, f"{prefix}e{int(chosen[t, n])}.", mlp["expert"]["limit"], low)[0]
    if mlp.get("shared"):
        out = out + clamped_expert(h, w, prefix + "shared.", mlp["shared"]["limit"], low)
    return out


MIXERS = {"parallel": parallel_mixer, "mlstm": mlstm_mixer, "mlstm_2": mlstm_mixer}


def forward(config, w, tokens, dtype=torch.float64, low=None, return_layers=False, margins=None):
    """Logits [T, vocab] of a whole sequence (and the residual stream after every layer).  ``margins``: a list
    that receives every layer's routing margins (see ``routed_experts``)."""
    tokens = torch.as_tensor(tokens, dtype=torch.long)
    eps = config["norm"]["eps"]
    x = w["embed"][tokens].to(dtype) + w["pos"][:len(tokens)].to(dtype)
    after = []
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}."
        h = _round(scalar_norm(x, w[p + "norm1"], eps), low)
        branch = MIXERS[layer["type"]](h, w, p + "mix.", layer["mixer"], eps, low)
        if layer.get("mlp") is not None:
            branch = branch + routed_experts(h, w, p + "mlp.", layer["mlp"], low, margins)
        x = x + branch
        after.append(x.clone())
    h = _round(scalar_norm(x, w["final.norm"], eps), low)
    logits = h @ w["head"].to(dtype).t()
    cap = config.get("logit_softcap")
    if cap:
        logits = capped(logits, cap)
    return (logits, torch.stack(after)) if return_layers else logits
