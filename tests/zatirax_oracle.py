"""Plain, slow restatement of the Zatirax decoder for the tests: one function per mechanism, one
sequence at a time, float64 throughout (angles included), nothing imported from the package under
test.

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


def norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * f64(weight)


# ------------------------------------------------------------------------------ positions
def stretched(f, scaling):
    """One rotary frequency under a context extension: long wavelengths are divided by the
    factor, short ones kept, those between interpolated."""
    if scaling is None:
        return f
    wavelength, old = 2.0 * math.pi / f, scaling["original"]
    if wavelength < old / scaling["high"]:
        return f
    if wavelength > old / scaling["low"]:
        return f / scaling["factor"]
    s = (old / wavelength - scaling["low"]) / (scaling["high"] - scaling["low"])
    return (1.0 - s) * f / scaling["factor"] + s * f


def frequencies(rot):
    d = rot["dims"]
    return [stretched(rot["base"] ** (-2.0 * i / d), rot.get("scaling")) for i in range(d // 2)]


def rotate(x, positions, rot):
    """x [n, d]: the pairs (i, i + dims / 2) turned by their positions' angles, the dimensions
    from rot.dims on left alone."""
    n, half = rot["dims"], rot["dims"] // 2
    a = positions.double().unsqueeze(1) * torch.tensor(frequencies(rot), dtype=torch.float64)
    u, v = x[:, :half], x[:, half:n]
    return torch.cat([u * a.cos() - v * a.sin(), v * a.cos() + u * a.sin(), x[:, n:]], 1)


# ------------------------------------------------------------------------------ visibility
def in_window(i, j, size):
    return 0 <= i - j < size


def in_chunk(i, j, size):
    return j <= i and i // size == j // size


@functools.lru_cache(maxsize=64)
def visible(seen, n, size):
    return torch.tensor([[seen(i, j, size) for j in range(n)] for i in range(n)], dtype=torch.bool)


def weights_of(scores, mask, sink=None):
    """Softmax over the visible keys; ``sink``: a further term of the denominator."""
    s = scores.masked_fill(~mask, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.clamp(top, min=float(sink))
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(f64(sink) - top)
    return e / total


# ------------------------------------------------------------------------------ mixers
def latent_attention(h, m, w, p, eps):
    H, d, r, dv, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    n = h.shape[0]
    pos = torch.arange(n)
    q = apply(w[p + "q"], h)
    kv = apply(w[p + "dkv"], h)
    c = norm(kv[:, :rank], w[p + "dkv.norm"], eps)
    shared = rotate(kv[:, rank:], pos, m["rot"])
    k, v = apply(w[p + "uk"], c), apply(w[p + "uv"], c)
    mask = visible(in_window, n, m["mask"]["size"])
    outs = []
    for a in range(H):
        qa = q[:, a * (d + r):(a + 1) * (d + r)]
        s = qa[:, :d] @ k[:, a * d:(a + 1) * d].t() + rotate(qa[:, d:], pos, m["rot"]) @ shared.t()
        outs.append(weights_of(s * m["scale"], mask) @ v[:, a * dv:(a + 1) * dv])
    return apply(w[p + "o"], torch.cat(outs, 1))


def gated_output(o, h, w_gate):
    return o / (1.0 + torch.exp(-apply(w_gate, h)))


def attention(h, m, w, p, eps):
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    n = h.shape[0]
    pos = torch.arange(n)
    q, k, v = (apply(w[p + x], h) for x in ("q", "k", "v"))
    mask = visible(in_chunk, n, m["mask"]["size"])
    ready = lambda x, weight: rotate(norm(x, weight, eps), pos, m["rot"])
    outs = []
    for a in range(H):
        g = a // (H // G)
        qa = ready(q[:, a * d:(a + 1) * d], w[p + "q.norm"])
        ka = ready(k[:, g * d:(g + 1) * d], w[p + "k.norm"])
        s = qa @ ka.t() * m["scale"]
        outs.append(weights_of(s, mask, f64(w[p + "sink"])[a]) @ v[:, g * dv:(g + 1) * dv])
    return apply(w[p + "o"], gated_output(torch.cat(outs, 1), h, w[p + "g"]))


def mix(kind, *a):
    return latent_attention(*a) if kind == "latent_attention" else attention(*a)


# ------------------------------------------------------------------------------ feed-forward
def clamped_swish(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g / (1.0 + torch.exp(-1.702 * g)) * (u + 1.0)


def feed_forward(h, f, w, p):
    return apply(w[p + "down"], clamped_swish(apply(w[p + "gate"], h), apply(w[p + "up"], h),
                                              f["limit"]))


# ------------------------------------------------------------------------------ the model
def runs(cfg):
    """(layer, step vector to add before it or None) in the order of execution."""
    loop = cfg.get("loop")
    order = []
    for i in range(len(cfg["layers"])):
        if loop and i == loop["start"]:
            for t in range(loop["times"]):
                order += [(j, t if j == loop["start"] else None)
                          for j in range(loop["start"], loop["stop"])]
        elif not loop or not loop["start"] <= i < loop["stop"]:
            order.append((i, None))
    return order


def layer(x, spec, w, p, eps):
    x = x + norm(mix(spec["type"], norm(x, w[p + "norm1"], eps), spec["mixer"], w, p + "mix.", eps),
                 w[p + "norm1b"], eps)
    if spec.get("mlp") is not None:
        x = x + norm(feed_forward(norm(x, w[p + "norm2"], eps), spec["mlp"], w, p + "mlp."),
                     w[p + "norm2b"], eps)
    return x


def forward(cfg, w, tokens, layers_out=None):
    """Logits [n, vocab] of one whole sequence; ``layers_out`` (a list) receives the residual
    stream after every layer run."""
    eps = cfg["norm"]["eps"]
    x = f64(w["embed"])[torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, t in runs(cfg):
        if t is not None:
            x = x + f64(w["loop.step"])[t]
        x = layer(x, cfg["layers"][i], w, "l%d." % i, eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return apply(w["head"], norm(x, w["final.norm"], eps))
