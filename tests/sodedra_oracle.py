"""A plain, slow Sodedra: one function per mechanism, one token or one head at a time, whole sequences, no cache.

Everything runs in the dtype of the weights handed in (the tests use float64).  Nothing here is shared with the
package: the equations are written out again, in loops where a loop says it most directly.
Shapes: a sequence is x [T, width]; heads are [T, heads, dim].
"""
import math

import torch

# With a generator here every projection's input and output is multiplied by 1 + 2^-9 randn: what rounding activations
# to bfloat16 does to an answer.
NOISE = None


def linear(x, w, b=None):
    if NOISE is None:
        y = x @ w.T
        return y if b is None else y + b
    jitter = lambda t: t * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=NOISE, dtype=t.dtype))
    y = jitter(x) @ w.T
    return jitter(y if b is None else y + b)


# ------------------------------------------------------------------------------------------- mechanisms
def unit_rms(x, eps):
    """x over its root mean square along the last dimension, eps inside the root."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return unit_rms(x, eps) * (1.0 + w)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def log_sigmoid(z):
    return -softplus(-z)


def frequencies(base, dims, scaling):
    """Rotary frequencies in float64; long wavelengths divided by a factor, a ramp in between."""
    f = []
    for i in range(dims // 2):
        w = base ** (-2.0 * i / dims)
        if scaling:
            length = 2.0 * math.pi / w
            orig, lo, hi, factor = (float(scaling[k]) for k in ("original", "low", "high", "factor"))
            if length > orig / lo:
                w = w / factor
            elif length >= orig / hi:
                s = (orig / length - lo) / (hi - lo)
                w = (1.0 - s) * w / factor + s * w
        f.append(w)
    return f


def rotate(x, base, dims, scaling=None, first_position=0):
    """Rotary positions on the first `dims` of every head of x [T, heads, dim], i paired with i + dims/2."""
    y = x.clone()
    position = first_position + torch.arange(x.shape[0], dtype=torch.float64)
    half = dims // 2
    for i, f in enumerate(frequencies(base, dims, scaling)):
        a = position * f
        c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i] = u * c - v * s
        y[:, :, i + half] = v * c + u * s
    return y


def window_attention(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query i of head h sees keys i - window + 1 .. i of head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[-1])
    i = torch.arange(T)
    back = i[:, None] - i[None, :]
    hidden = (back < 0) | (back >= window)
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(hidden, -math.inf)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (p / p.sum(-1, keepdim=True)) @ v[:, g]
    return out


def short_conv(x, w):
    """Causal convolution per channel: x [T, C], w [C, taps], the last column belongs to the current token."""
    y = torch.zeros_like(x)
    taps = w.shape[1]
    for t in range(x.shape[0]):
        for j in range(taps):
            if t - j >= 0:
                y[t] += x[t - j] * w[:, taps - 1 - j]
    return y


def delta_rule(q, k, v, beta, decay):
    """Token by token from S = 0: S <- decay * S (rows are key channels), u = beta (v - S^T k), S <- S + k u^T,
    o = S^T q.  q, k, decay [T, H, dk]; v [T, H, dv]; beta [T, H]."""
    T, H, dk = q.shape
    S = q.new_zeros(H, dk, v.shape[-1])
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        S = decay[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def stabilised_memory(q, k, v, i, f):
    """Exponentially gated matrix memory, token by token, with a running maximum that starts at 0.
    q, k [T, H, dk]; v [T, H, dv]; log gates i, f [T, H]."""
    T, H, dk = q.shape
    S, n, m = q.new_zeros(H, dk, v.shape[-1]), q.new_zeros(H, dk), q.new_zeros(H)
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        bottom = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = (S * q[t][:, :, None]).sum(1) / bottom[:, None]
    return out


def route(z, correction, top, groups, keep, scale):
    """Router logits z [T, E] -> (expert ids [T, top], weights [T, top]), one token at a time."""
    T, E = z.shape
    ids, ws = [], []
    for t in range(T):
        e = torch.exp(z[t] - z[t].max())
        s = e / e.sum()
        choice = s + correction
        size = E // groups
        best = [float(choice[g * size:(g + 1) * size].max()) for g in range(groups)]
        allowed = sorted(range(groups), key=lambda g: -best[g])[:keep]
        order = sorted((x for x in range(E) if x // size in allowed), key=lambda x: -float(choice[x]))[:top]
        w = s[order]
        ids.append(order)
        ws.append(w / (w.sum() + 1e-20) * scale)
    return torch.tensor(ids), torch.stack(ws)


# ------------------------------------------------------------------------------------------- sublayers
def attention(h, w, cfg, eps):
    T, H, G, d, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    rot = cfg["rot"]
    q = rotate(linear(h, w["q"], w["q.b"]).view(T, H, d), rot["base"], rot["dims"], rot.get("scaling"))
    k = rotate(linear(h, w["k"], w["k.b"]).view(T, G, d), rot["base"], rot["dims"], rot.get("scaling"))
    v = linear(h, w["v"], w["v.b"]).view(T, G, dv)
    o = window_attention(q, k, v, cfg["scale"], cfg["mask"]["size"]).reshape(T, H * dv)
    return linear(o * sigmoid(linear(h, w["g"])), w["o"])


def channel_delta(h, w, cfg, eps):
    T, H, G, dk, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (silu(short_conv(linear(h, w[n]), w[n + ".conv"])) for n in "qkv")
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q = unit(q.view(T, G, dk)) * dk ** -0.5
    k = unit(k.view(T, G, dk))
    pick = torch.arange(H) // (H // G)
    beta = sigmoid(linear(h, w["b"]))
    step = softplus(linear(h, w["a1"]) @ w["a2"].T + w["dt_bias"]).view(T, H, dk)
    decay = torch.exp(-torch.exp(w["A_log"])[None, :, None] * step)
    o = unit_rms(delta_rule(q[:, pick], k[:, pick], v.view(T, H, dv), beta, decay), eps) * w["norm"]
    gate = sigmoid(linear(linear(h, w["g1"]), w["g2"]))
    return linear(o.reshape(T, H * dv) * gate, w["o"])


def mlstm(h, w, cfg, eps):
    T, H, dk, dv, cap = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"], cfg["gate_cap"]
    q = linear(h, w["q"]).view(T, H, dk) * dk ** -0.5
    k = linear(h, w["k"]).view(T, H, dk)
    v = linear(h, w["v"]).view(T, H, dv)
    i = cap * torch.tanh((linear(h, w["i"]) + w["i.b"]) / cap)
    f = log_sigmoid(cap * torch.tanh((linear(h, w["f"]) + w["f.b"]) / cap))
    o = unit_rms(stabilised_memory(q, k, v, i, f), eps).reshape(T, H * dv) * w["norm"]
    return linear(o * sigmoid(linear(h, w["g"])), w["o"])


def dense_mlp(h, w):
    return linear(silu(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


def experts(h, w, cfg):
    r = cfg["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    ids, weights = route(linear(h, w["router"]), w["correction"], r["top"], g["count"], g["keep"], r["scale"])
    out = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = None
        for t, j in (ids == e).nonzero().tolist():
            if y is None:
                y = dense_mlp(h, _sub(w, f"e{e}."))
            out[t] += weights[t, j] * y[t]
    return out


MIXERS = {"attention": attention, "channel_delta": channel_delta, "mlstm": mlstm}


def _sub(w, prefix):
    return {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}


# ------------------------------------------------------------------------------------------- the model
def forward(tokens, config, weights, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  `layers_out`: a list that receives the residual after each layer."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{i}.")
        h = centred_norm(x, w["norm1"], eps)
        y = MIXERS[layer["type"]](h, _sub(w, "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            m = _sub(w, "mlp.")
            y = y + (experts(h, m, layer["mlp"]) if layer["mlp"]["kind"] == "moe" else dense_mlp(h, m))
        x = x + y
        if layers_out is not None:
            layers_out.append(x)
    return linear(centred_norm(x, weights["final.norm"], eps), weights["embed"])


def greedy(prompt, n, config, weights):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(toks, config, weights)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------- test models
def tensor_shapes(config, rank):
    """Name -> shape of every tensor of a model; `rank`: inner sizes (decay, gate) of the low-rank projections."""
    W, V = config["width"], config["vocab"]
    ra, rg = rank
    out = {"embed": (V, W), "final.norm": (W,)}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        x, H, dk, dv = p + "mix.", m["heads"], m["dim"], m["vdim"]
        G = m.get("kv_heads", H)
        out.update({p + "norm1": (W,), x + "q": ((G if layer["type"] == "channel_delta" else H) * dk, W), x + "k": (G * dk, W),
                    x + "o": (W, H * dv)})
        if layer["type"] == "attention":
            out.update({x + "v": (G * dv, W), x + "g": (H * dv, W), x + "q.b": (H * dk,), x + "k.b": (G * dk,),
                        x + "v.b": (G * dv,)})
        elif layer["type"] == "mlstm":
            out.update({x + "v": (H * dv, W), x + "g": (H * dv, W), x + "norm": (H * dv,), x + "i": (H, W), x + "i.b": (H,),
                        x + "f": (H, W), x + "f.b": (H,)})
        else:
            taps = m["conv"]
            out.update({x + "v": (H * dv, W), x + "q.conv": (G * dk, taps), x + "k.conv": (G * dk, taps),
                        x + "v.conv": (H * dv, taps), x + "b": (H, W), x + "A_log": (H,), x + "norm": (dv,), x + "a1": (ra, W),
                        x + "a2": (H * dk, ra), x + "dt_bias": (H * dk,), x + "g1": (rg, W), x + "g2": (H * dv, rg)})
        if layer["mlp"] is not None:
            kind, q = layer["mlp"]["kind"], p + "mlp."
            if kind == "dense":
                ffs = {q: layer["mlp"]["ff"]}
            else:
                E = layer["mlp"]["router"]["experts"]
                out.update({q + "router": (E, W), q + "correction": (E,)})
                ffs = {f"{q}e{e}.": layer["mlp"]["expert"]["ff"] for e in range(E)}
            for n, ff in ffs.items():
                out.update({n + "gate": (ff, W), n + "up": (ff, W), n + "down": (W, ff)})
    return out


def random_weights(config, rank=(6, 6), seed=0):
    """bfloat16 weights of a sensible scale: linear maps keep the variance, norms sit around one, decays near one."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config, rank).items():
        r = torch.randn(shape, generator=g)
        leaf = name.rsplit("mix.", 1)[-1]
        if leaf == "norm":
            t = 1.0 + 0.2 * r
        elif leaf == "dt_bias":
            t = -4.0 + 1.5 * r
        elif leaf == "A_log":
            t = 0.5 * r
        elif leaf == "f.b":
            t = 3.0 + r
        elif leaf == "i.b":
            t = -1.0 + r
        elif name.endswith("correction"):
            t = 0.3 * r
        elif len(shape) == 1:
            t = 0.2 * r
        elif name == "embed":
            t = r * 0.5
        elif name.endswith(".conv"):
            t = r * 0.4
            t[:, -1] += 0.7
        else:
            t = r * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
