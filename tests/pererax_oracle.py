"""Plain, slow restatement of the Pererax decoder for the tests: one function per mechanism, one
sequence at a time and the recurrences token by token, float64 throughout, nothing imported from
the package under test.

``cfg`` is the dictionary of a checkpoint's config.json, ``w`` a dictionary of tensors under the
checkpoint's names.
"""

import functools
import math

import torch


def f64(t):
    return t.detach().cpu().to(torch.float64)


def apply(w, x):
    """A linear map stored [out, in] on every row of x."""
    return x @ f64(w).t()


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, weight, eps):
    return rms(x, eps) * f64(weight)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------------------ positions
def rotate(x, positions, rot):
    """x [n, d]: the pairs (i, i + dims / 2) turned by their positions' angles, the dimensions
    from rot.dims on left alone."""
    n, half = rot["dims"], rot["dims"] // 2
    f = torch.tensor([rot["base"] ** (-2.0 * i / n) for i in range(half)], dtype=torch.float64)
    a = positions.double().unsqueeze(1) * f
    u, v = x[:, :half], x[:, half:n]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), x[:, n:]], 1)


# ------------------------------------------------------------------------------ attention
def sees(i, j, size):
    """Whether position i attends to j; size None: no window."""
    return j <= i and (size is None or i - j < size)


@functools.lru_cache(maxsize=64)
def visible(seen, n, size):
    return torch.tensor([[seen(i, j, size) for j in range(n)] for i in range(n)], dtype=torch.bool)


def weights_of(scores, mask, sink):
    """Softmax over the visible keys; ``sink``: one more term exp(0) in the denominator."""
    s = scores.masked_fill(~mask, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink:
        top = torch.clamp(top, min=0.0)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    return e / (total + torch.exp(-top) if sink else total)


def capped(scores, cap):
    return cap * torch.tanh(scores / cap)


def projection_norm(x, weight, eps):
    """The norm of queries (or keys): over all heads' rows at once."""
    return norm(x, weight, eps)


def heads_of_queries(h, m, w, p, eps):
    """Scores [H, n, n] of the rows of h and the raw key projection."""
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(h.shape[0])
    raw = apply(w[p + "k"], h)
    q = projection_norm(apply(w[p + "q"], h), w[p + "q.norm"], eps)
    k = projection_norm(raw, w[p + "k.norm"], eps)
    out = []
    for a in range(H):
        g = a // (H // G)
        qa = rotate(q[:, a * d:(a + 1) * d], pos, m["rot"])
        ka = rotate(k[:, g * d:(g + 1) * d], pos, m["rot"])
        out.append(qa @ ka.t() * m["scale"])
    return torch.stack(out), raw


def weighted_values(weights, v, m, dv):
    H, G = m["heads"], m["kv_heads"]
    return torch.cat([weights[a] @ v[:, (a // (H // G)) * dv:(a // (H // G) + 1) * dv]
                      for a in range(H)], 1)


def window_attention(h, m, w, p, eps):
    """Sliding window; the values are the keys as projected."""
    s, raw = heads_of_queries(h, m, w, p, eps)
    pr = weights_of(s, visible(sees, h.shape[0], m["mask"]["size"]), False)
    return apply(w[p + "o"], weighted_values(pr, raw, m, m["dim"]))


def capped_attention(h, m, w, p, eps):
    """Causal, scores capped, a sink with score 0."""
    s, _ = heads_of_queries(h, m, w, p, eps)
    pr = weights_of(capped(s, m["softcap"]), visible(sees, h.shape[0], None), True)
    return apply(w[p + "o"], weighted_values(pr, apply(w[p + "v"], h), m, m["vdim"]))


# ------------------------------------------------------------------------------ matrix memory
def memory_gates(zi, zf, cap):
    """(log input gate, log forget gate)."""
    i = cap * torch.tanh(zi / cap)
    f = cap * torch.tanh(zf / cap)
    return i, -softplus(-f)


def memory_scan(q, k, v, i, f):
    """One head: q, k [n, d], v [n, dv], log gates i, f [n] -> [n, dv]."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=torch.float64)
    z = torch.zeros(k.shape[1], dtype=torch.float64)
    m, out = torch.zeros((), dtype=torch.float64), []
    for t in range(k.shape[0]):
        new = torch.maximum(f[t] + m, i[t])
        keep, put = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep * S + put * torch.outer(k[t], v[t])
        z = keep * z + put * k[t]
        m = new
        out.append(S.t() @ q[t] / (torch.maximum((z @ q[t]).abs(), torch.exp(-m)) + 1e-6))
    return torch.stack(out)


def matrix_memory(h, m, w, p, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, k, v = apply(w[p + "q"], h) * d ** -0.5, apply(w[p + "k"], h), apply(w[p + "v"], h)
    i, f = memory_gates(apply(w[p + "i"], h) + f64(w[p + "i.b"]),
                        apply(w[p + "f"], h) + f64(w[p + "f.b"]), m["gate_cap"])
    o = torch.cat([rms(memory_scan(q[:, a * d:(a + 1) * d], k[:, a * d:(a + 1) * d],
                                   v[:, a * dv:(a + 1) * dv], i[:, a], f[:, a]), eps)
                   for a in range(H)], 1)
    return apply(w[p + "o"], o * f64(w[p + "norm"]) * sigmoid(apply(w[p + "g"], h)))


def parallel(h, m, w, p, eps):
    left = norm(capped_attention(h, m["left"], w, p + "left.", eps), w[p + "left.out"], eps)
    right = norm(matrix_memory(h, m["right"], w, p + "right.", eps), w[p + "right.out"], eps)
    return 0.5 * (left + right)


# ------------------------------------------------------------------------------ delta rule
def short_conv(x, taps):
    """Causal convolution per channel over time, the last column for the current token; silu."""
    n, width = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(width - 1, x.shape[1], dtype=torch.float64), x])
    c = f64(taps)
    return silu(sum(padded[j:j + n] * c[:, j] for j in range(width)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def decays(z, a_log, dt_bias, heads):
    """[n, heads, dim]: the factor of every key channel's row of the state."""
    z = softplus(z + f64(dt_bias)).reshape(z.shape[0], heads, -1)
    return torch.exp(-torch.exp(f64(a_log)).view(heads, 1) * z)


def delta_scan(q, k, v, g, beta):
    """One head: q, k, g [n, d], v [n, dv], beta [n] -> [n, dv]."""
    S, out = torch.zeros(k.shape[1], v.shape[1], dtype=torch.float64), []
    for t in range(k.shape[0]):
        S = g[t].unsqueeze(1) * S
        u = beta[t] * (v[t] - S.t() @ k[t])
        S = S + torch.outer(k[t], u)
        out.append(S.t() @ q[t])
    return torch.stack(out)


def channel_delta(h, m, w, p, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(apply(w[p + x], h), w[p + x + ".conv"]) for x in ("q", "k", "v"))
    beta = sigmoid(apply(w[p + "b"], h))
    g = decays(apply(w[p + "a2"], apply(w[p + "a1"], h)), w[p + "A_log"], w[p + "dt_bias"], H)
    outs = []
    for a in range(H):
        b = a // (H // G)
        o = delta_scan(unit(q[:, b * d:(b + 1) * d]) * d ** -0.5, unit(k[:, b * d:(b + 1) * d]),
                       v[:, a * dv:(a + 1) * dv], g[:, a], beta[:, a])
        outs.append(norm(o, w[p + "norm"], eps))
    gate = sigmoid(apply(w[p + "g2"], apply(w[p + "g1"], h)))
    return apply(w[p + "o"], torch.cat(outs, 1) * gate)


MIXERS = {"channel_delta": channel_delta, "parallel": parallel, "attention": window_attention}


# ------------------------------------------------------------------------------ feed-forward
def clamped_swish(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert(h, w, p, limit):
    return apply(w[p + "down"], clamped_swish(apply(w[p + "gate"], h), apply(w[p + "up"], h), limit))


def route(h, w_router, correction, top, scale):
    """(chosen outputs [n, top], their weights, how far the last chosen one is ahead)."""
    z = apply(w_router, h)
    s = torch.exp(z - z.max(-1, keepdim=True).values)
    s = s / s.sum(-1, keepdim=True)
    order = torch.sort(s + f64(correction), dim=-1, descending=True, stable=True)
    chosen = order.indices[:, :top]
    lead = order.values[:, top - 1] - order.values[:, top] if top < z.shape[1] else \
        torch.full((h.shape[0],), math.inf, dtype=torch.float64)
    return chosen, s.gather(1, chosen) * scale, lead


def mixture(h, f, w, p, margins=None):
    r, limit = f["router"], f["expert"]["limit"]
    chosen, weight, lead = route(h, w[p + "router"], w[p + "correction"], r["top"], r["scale"])
    if margins is not None:
        margins.append(lead)
    out = torch.zeros_like(h)
    for e in range(r["experts"] + r["identity"]):
        t, j = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            y = h[t] if e >= r["experts"] else expert(h[t], w, "%se%d." % (p, e), limit)
            out[t] += weight[t, j].unsqueeze(1) * y
    if f.get("shared"):
        out = out + expert(h, w, p + "shared.", f["shared"]["limit"])
    return out


# ------------------------------------------------------------------------------ the model
def residual(x, y, weight, scale, eps):
    """The norm and the layer scale lie on the sublayer's output."""
    return x + norm(y, weight, eps) * f64(scale)


def weights_index(cfg, i):
    """The layer whose tensors layer i uses."""
    src = cfg["layers"][i].get("weights_of")
    return i if src is None else weights_index(cfg, src)


def layer(x, spec, w, p, eps, margins=None):
    y = MIXERS[spec["type"]](x, spec["mixer"], w, p + "mix.", eps)
    x = residual(x, y, w[p + "norm1"], w[p + "ls1"], eps)
    if spec.get("mlp") is not None:
        x = residual(x, mixture(x, spec["mlp"], w, p + "mlp.", margins), w[p + "norm2"],
                     w[p + "ls2"], eps)
    return x


def forward(cfg, w, tokens, layers_out=None, margins=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out`` (a list) receives the residual
    stream after every layer, ``margins`` each router's lead of the last chosen output."""
    eps = cfg["norm"]["eps"]
    x = f64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)]
    for i, spec in enumerate(cfg["layers"]):
        x = layer(x, spec, w, "l%d." % weights_index(cfg, i), eps, margins)
        if layers_out is not None:
            layers_out.append(x.clone())
    return apply(w["embed"], norm(x, w["final.norm"], eps))
