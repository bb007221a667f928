"""Plain, slow restatement of the Taralix decoder for the tests: one function per mechanism, one
sequence at a time, float64 throughout, nothing imported from the package under test.

``cfg`` is the dictionary of a checkpoint's config.json, ``w`` a dictionary of tensors under the
checkpoint's names.
"""

import math

import torch


def f64(t):
    return t.detach().cpu().to(torch.float64)


def rms(x, eps):
    """x divided by its root mean square (eps under the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, weight, eps):
    """RMS norm whose stored weight is the deviation from one."""
    return rms(x, eps) * (1.0 + f64(weight))


def plain_norm(x, weight, eps):
    return rms(x, eps) * f64(weight)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z / (1.0 + torch.exp(-z))


def apply(w, x):
    """A linear map stored [out, in] on every row of x."""
    return x @ f64(w).t()


def latent(h, w_dkv, w_norm, eps):
    """What a layer keeps per token: the normalised projection to kv_rank dimensions."""
    return plain_norm(apply(w_dkv, h), w_norm, eps)


def attend_latent(h, c, w_q, w_uk, w_uv, w_o, heads, dim, vdim, scale):
    """Causal softmax attention of the rows of h over the latents c of the whole sequence (the
    rows of h are its last ones). Keys and values are expanded head by head."""
    n, total = h.shape[0], c.shape[0]
    q = apply(w_q, h)
    k = apply(w_uk, c)
    v = apply(w_uv, c)
    outs = []
    for a in range(heads):
        qa = q[:, a * dim:(a + 1) * dim]
        ka = k[:, a * dim:(a + 1) * dim]
        va = v[:, a * vdim:(a + 1) * vdim]
        s = qa @ ka.t() * scale
        for i in range(n):
            s[i, total - n + i + 1:] = -math.inf
        s = s - s.max(-1, keepdim=True).values
        p = torch.exp(s)
        outs.append((p / p.sum(-1, keepdim=True)) @ va)
    return apply(w_o, torch.cat(outs, -1))


def gated(h, w_gate, w_up, w_down, act):
    return apply(w_down, act(apply(w_gate, h)) * apply(w_up, h))


def route(h, w_router, bias, top):
    """(chosen experts [n, top], their weights): softmax over the chosen logits only."""
    z = apply(w_router, h) + f64(bias)
    chosen = torch.argsort(z, dim=-1, descending=True, stable=True)[:, :top]
    zc = z.gather(1, chosen)
    e = torch.exp(zc - zc.max(-1, keepdim=True).values)
    return chosen, e / e.sum(-1, keepdim=True)


def route_margin(h, w_router, bias, top):
    """Per token, how far the last chosen logit lies above the first one left out."""
    z = torch.sort(apply(w_router, h) + f64(bias), dim=-1, descending=True).values
    if top == z.shape[1]:
        return torch.full((h.shape[0],), math.inf, dtype=torch.float64)
    return z[:, top - 1] - z[:, top]


def mixture(h, w, prefix, top):
    chosen, weight = route(h, w[prefix + "router"], w[prefix + "router.b"], top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for j in range(top):
            p = "%se%d." % (prefix, int(chosen[t, j]))
            out[t] += weight[t, j] * gated(h[t:t + 1], w[p + "gate"], w[p + "up"], w[p + "down"],
                                           silu)[0]
    return out


def forward(cfg, w, tokens, layers_out=None, margins=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out`` (a list) receives the residual
    stream after every layer, ``margins`` each router's ``route_margin``."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = f64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)]
    latents = {}
    for i, spec in enumerate(cfg["layers"]):
        m, p = spec["mixer"], "l%d." % i
        src = m.get("kv_from")
        if src is None:
            latents[i] = latent(x, w[p + "mix.dkv"], w[p + "mix.dkv.norm"], eps)
            src = i
        y = attend_latent(x, latents[src], w[p + "mix.q"], w[p + "mix.uk"], w[p + "mix.uv"],
                          w[p + "mix.o"], m["heads"], m["dim"], m["vdim"], m["scale"])
        x = zero_centred_norm(alpha * x + y, w[p + "norm1"], eps)
        f = spec.get("mlp")
        if f is not None:
            if f["kind"] == "dense":
                y = gated(x, w[p + "mlp.gate"], w[p + "mlp.up"], w[p + "mlp.down"], gelu_tanh)
            else:
                if margins is not None:
                    margins.append(route_margin(x, w[p + "mlp.router"], w[p + "mlp.router.b"],
                                                f["router"]["top"]))
                y = mixture(x, w, p + "mlp.", f["router"]["top"])
            x = zero_centred_norm(alpha * x + y, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return apply(w["head"], zero_centred_norm(x, w["final.norm"], eps))
