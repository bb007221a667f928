"""Plain, slow restatement of the Pefivik decoder for the tests: one function per mechanism, one
sequence at a time and the recurrence token by token, float64 throughout, nothing imported from the
package under test.

``cfg`` is the dictionary of a checkpoint's config.json, ``w`` a dictionary of tensors under the
checkpoint's names.
"""

import math

import torch


def f64(t):
    return t.detach().cpu().to(torch.float64)


def apply(w, x):
    """A linear map stored [out, in] on every row of x."""
    return x @ f64(w).t()


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def stream_norm(x, gain, eps):
    """Norm of the residual stream: one number for all coordinates."""
    return rms(x, eps) * f64(gain)


# ------------------------------------------------------------------------------ embedding
def bigram_rows(tokens, b):
    """Row of the bigram table of every token; the last row where there is no previous token."""
    rows = [b["buckets"]]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((prev * b["mul_prev"] + cur * b["mul_cur"]) % b["buckets"])
    return rows[:len(tokens)]


def embedding(cfg, w, tokens):
    rows = bigram_rows(list(tokens), cfg["embedding"]["bigram"])
    return f64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)] + f64(w["bigram"])[rows]


# ------------------------------------------------------------------------------ latent attention
def sees(i, j):
    return j <= i


def weights_of(scores, sink):
    """scores [n, n] of one head, softmax over the visible keys with one further term exp(sink) in
    the denominator."""
    n = scores.shape[0]
    mask = torch.tensor([[sees(i, j) for j in range(n)] for i in range(n)], dtype=torch.bool)
    s = scores.masked_fill(~mask, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=sink)
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + math.exp(sink) * torch.exp(-top))


def latent(h, w, p, eps):
    return rms(apply(w[p + "dkv"], h), eps) * f64(w[p + "dkv.norm"])


def head_gates(h, w, p):
    """[n, H]: one factor per head."""
    return sigmoid(apply(w[p + "g"], h))


def latent_attention(h, m, w, p, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, c = apply(w[p + "q"], h), latent(h, w, p, eps)
    k, v = apply(w[p + "uk"], c), apply(w[p + "uv"], c)
    g = head_gates(h, w, p)
    out = []
    for a in range(H):
        s = q[:, a * d:(a + 1) * d] @ k[:, a * d:(a + 1) * d].t() * m["scale"]
        pr = weights_of(s, float(w[p + "sink"][a]))
        out.append(pr @ v[:, a * dv:(a + 1) * dv] * g[:, a:a + 1])
    return apply(w[p + "o"], torch.cat(out, 1))


# ------------------------------------------------------------------------------ hgrn2
def forget_gates(z, lower):
    l = f64(lower)
    return l + (1.0 - l) * sigmoid(z)


def hgrn2_scan(q, f, v):
    """One head: q, f [n, d], v [n, dv] -> [n, dv]."""
    S, out = torch.zeros(q.shape[1], v.shape[1], dtype=torch.float64), []
    for t in range(q.shape[0]):
        S = f[t].unsqueeze(1) * S + torch.outer(1.0 - f[t], v[t])
        out.append(S.t() @ q[t])
    return torch.stack(out)


def hgrn2(h, m, w, p, eps):
    H, d, dv = m["heads"], m["dim"], m["vdim"]
    q, v = silu(apply(w[p + "q"], h)), apply(w[p + "v"], h)
    f = forget_gates(apply(w[p + "f"], h) + f64(w[p + "f.b"]), w[p + "lower"])
    out = []
    for a in range(H):
        o = hgrn2_scan(q[:, a * d:(a + 1) * d], f[:, a * d:(a + 1) * d], v[:, a * dv:(a + 1) * dv])
        out.append(rms(o, eps) * f64(w[p + "norm"]))
    return apply(w[p + "o"], torch.cat(out, 1))


MIXERS = {"latent_attention": latent_attention, "hgrn2": hgrn2}


# ------------------------------------------------------------------------------ feed-forward
def poly_norm(z, act, eps):
    a, b, c, e = (float(x) for x in act)
    return a * rms(z, eps) + b * rms(z ** 2, eps) + c * rms(z ** 3, eps) + e


def dense(h, f, w, p, eps):
    z = apply(w[p + "up"], h) + f64(w[p + "up.b"])
    return apply(w[p + "down"], poly_norm(z, w[p + "act"], eps)) + f64(w[p + "down.b"])


def expert(h, w, p):
    return apply(w[p + "down"], silu(apply(w[p + "gate"], h)) * apply(w[p + "up"], h))


def route(h, w_router, r):
    """(chosen experts [n, top], their weights, how close the choice was: the smaller of the leads of
    the last kept group and of the last chosen expert)."""
    s = sigmoid(apply(w_router, h))
    n, E = s.shape
    count, keep, top = r["groups"]["count"], r["groups"]["keep"], r["top"]
    best_two = torch.sort(s.view(n, count, E // count), dim=-1, descending=True).values[..., :2].sum(-1)
    groups = torch.sort(best_two, dim=-1, descending=True, stable=True)
    lead = torch.full((n,), math.inf, dtype=torch.float64)
    if keep < count:
        lead = groups.values[:, keep - 1] - groups.values[:, keep]
    allowed = torch.zeros(n, count, dtype=torch.bool).scatter_(1, groups.indices[:, :keep], True)
    allowed = allowed.repeat_interleave(E // count, 1)
    order = torch.sort(s.masked_fill(~allowed, -math.inf), dim=-1, descending=True, stable=True)
    chosen = order.indices[:, :top]
    if top < keep * (E // count):
        lead = torch.minimum(lead, order.values[:, top - 1] - order.values[:, top])
    own = s.gather(1, chosen)
    return chosen, own / (own.sum(-1, keepdim=True) + 1e-20) * r["scale"], lead


def mixture(h, f, w, p, margins=None):
    chosen, weight, lead = route(h, w[p + "router"], f["router"])
    if margins is not None:
        margins.append(lead)
    out = expert(h, w, p + "shared.") if f.get("shared") else torch.zeros_like(h)
    for e in range(f["router"]["experts"]):
        t, j = torch.nonzero(chosen == e, as_tuple=True)
        if t.numel():
            out[t] += weight[t, j].unsqueeze(1) * expert(h[t], w, "%se%d." % (p, e))
    return out


# ------------------------------------------------------------------------------ the model
def order_of_runs(cfg):
    """(layer, pass it begins or None) one after the other."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, None) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    out = [(i, None) for i in range(a)]
    for t in range(loop["times"]):
        out += [(i, t if i == a else None) for i in range(a, b)]
    return out + [(i, None) for i in range(b, n)]


def enter_pass(x, x0, steps, t):
    """What happens to the stream ahead of pass t."""
    return x + (x0 if t > 0 else 0.0) + f64(steps)[t]


def residual(x, y, m):
    return x + m * y


def layer(x, spec, w, p, cfg, margins=None):
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    h = stream_norm(x, w[p + "norm1"], eps)
    x = residual(x, MIXERS[spec["type"]](h, spec["mixer"], w, p + "mix.", eps), m)
    f = spec.get("mlp")
    if f is not None:
        h = stream_norm(x, w[p + "norm2"], eps)
        y = dense(h, f, w, p + "mlp.", eps) if f["kind"] == "dense" else \
            mixture(h, f, w, p + "mlp.", margins)
        x = residual(x, y, m)
    return x


def output(x, cfg, w):
    z = apply(w["head"], stream_norm(x, w["final.norm"], cfg["norm"]["eps"]))
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(z / cap)


def forward(cfg, w, tokens, layers_out=None, margins=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out`` (a list) receives the residual
    stream after every layer run, ``margins`` how close each router's choices were."""
    x = x0 = embedding(cfg, w, tokens)
    for i, t in order_of_runs(cfg):
        if t is not None:
            x = enter_pass(x, x0, w["loop.step"], t)
        x = layer(x, cfg["layers"][i], w, "l%d." % i, cfg, margins)
        if layers_out is not None:
            layers_out.append(x.clone())
    return output(x, cfg, w)
