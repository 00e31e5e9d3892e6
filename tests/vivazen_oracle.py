"""A plain, slow Vivazen: one function per mechanism, one head or one token at a time, whole sequences, no cache.

Everything runs in the dtype of the weights handed in (the tests use float64).  Nothing here is shared with the
package: the equations are written out again, in loops where a loop says it most directly.
Shapes: a sequence is x [T, width]; heads are [T, heads, dim].
"""
import math

import torch

# With a generator here every projection's input and output is multiplied by 1 + 2^-9 randn: what rounding activations
# to bfloat16 does to an answer.
NOISE = None


def jitter(t):
    return t if NOISE is None else t * (1 + 2.0 ** -9 * torch.randn(t.shape, generator=NOISE, dtype=t.dtype))


def linear(x, w):
    return jitter(jitter(x) @ w.T)


# ------------------------------------------------------------------------------------------- mechanisms
def rms_norm(x, w, eps):
    """x over its root mean square along the last dimension (eps inside the root), times w."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def grouped_norm(x, w, groups, eps):
    """Each of `groups` consecutive parts over its own root mean square; the whole times w."""
    n = x.shape[-1] // groups
    parts = [x[..., g * n:(g + 1) * n] for g in range(groups)]
    return torch.cat([p / torch.sqrt((p * p).mean(-1, keepdim=True) + eps) for p in parts], dim=-1) * w


def join(x, y, w, alpha, groups, eps):
    """The residual behind a sublayer: the weighted sum goes through the norm."""
    return grouped_norm(alpha * x + y, w, groups, eps)


def short_conv(x, w):
    """Causal convolution per channel: x [T, C], w [C, taps], the last column belongs to the current token."""
    y = torch.zeros_like(x)
    taps = w.shape[1]
    for back in range(taps):
        n = x.shape[0] - back
        if n > 0:
            y[back:] += x[:n] * w[:, taps - 1 - back]
    return y


def yarn_frequencies(rot):
    """Per pair the angle of one position, and the factor of cos and sin."""
    dims, base, s = rot["dims"], rot["base"], rot["scaling"]
    at = lambda turns: dims * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i in range(dims // 2):
        f = base ** (-2.0 * i / dims)
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate_pairs(x, rot, first_position=0):
    """Rotary positions on every head of x [T, heads, dims]: neighbours 2i and 2i + 1 turn together."""
    y = x.clone()
    freq, size = yarn_frequencies(rot)
    position = first_position + torch.arange(x.shape[0], dtype=torch.float64)
    for i, f in enumerate(freq):
        c, s = ((position * f).cos() * size).to(x.dtype)[:, None], ((position * f).sin() * size).to(x.dtype)[:, None]
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * c - v * s
        y[:, :, 2 * i + 1] = v * c + u * s
    return y


def visible(T, window=None):
    """[T, T]: may query i (row) see key j?  Inside the window (None: everything before it)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if window is None else i - j < window
    return (j <= i) & near


def softmax(s, mask, sink=None):
    """Over the visible keys of every row; a sink adds exp(sink) to the denominator."""
    s = s.masked_fill(~mask, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    if sink is not None:
        total = total + torch.exp(sink - top)
    return e / total


def sink_attention(q, k, v, scale, mask, sink):
    """q, k [T, H, d], v [T, H, dv], sink [H]."""
    out = q.new_zeros(q.shape[0], q.shape[1], v.shape[-1])
    for h in range(q.shape[1]):
        out[:, h] = softmax((q[:, h] @ k[:, h].T) * scale, mask, sink[h]) @ v[:, h]
    return out


def talking_attention(q, k, v, scale, softcap, talk):
    """q [T, H, d], k [T, G, d], v [T, G, dv], talk [H, H]: softly capped causal attention whose heads' weights are mixed
    before they meet the values."""
    T, H, _ = q.shape
    G = k.shape[1]
    mask = visible(T)
    p = []
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        p.append(softmax(softcap * torch.tanh(s / softcap), mask))
    out = q.new_zeros(T, H, v.shape[-1])
    p = torch.stack(p)
    for h in range(H):
        mixed = (talk[h][:, None, None] * p).sum(0)
        out[:, h] = mixed @ v[:, h // (H // G)]
    return out


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


# ------------------------------------------------------------------------------------------- sublayers
def attention_mixer(h, w, cfg, eps):
    T, H, G, d, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (short_conv(linear(h, w[n]), w[n + ".conv"]) for n in "qkv")
    q = rms_norm(q, w["q.norm"], eps).view(T, H, d)
    k = rms_norm(k, w["k.norm"], eps).view(T, G, d)
    v = rms_norm(v.view(T, G, dv), 1.0, eps)
    o = talking_attention(jitter(q), jitter(k), jitter(v), cfg["scale"], cfg["softcap"], w["talk"])
    return linear(o.reshape(T, H * dv), w["o"])


def latent_mixer(h, w, cfg, eps):
    T, H, d, r, dv, rank = h.shape[0], cfg["heads"], cfg["dim"], cfg["rot_dim"], cfg["vdim"], cfg["kv_rank"]
    q = linear(h, w["q"]).view(T, H, d + r)
    both = linear(h, w["dkv"])
    c = rms_norm(both[:, :rank], w["dkv.norm"], eps)
    shared = jitter(rotate_pairs(both[:, rank:].view(T, 1, r), cfg["rot"]))
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], cfg["rot"])], dim=-1)
    k = torch.cat([linear(c, w["uk"]).view(T, H, d), shared.expand(T, H, r)], dim=-1)
    v = linear(c, w["uv"]).view(T, H, dv)
    o = sink_attention(jitter(q), k, v, cfg["scale"], visible(T, cfg["mask"]["size"]), w["sink"])
    o = o / (1.0 + torch.exp(-linear(h, w["g"])))[:, :, None]
    return linear(o.reshape(T, H * dv), w["o"])


def feed_forward(h, w):
    return linear(gelu_tanh(linear(h, w["gate"])) * linear(h, w["up"]), w["down"])


MIXERS = {"attention": attention_mixer, "latent_attention": latent_mixer}


def _sub(w, prefix):
    return {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}


def owner(config, i):
    """The layer whose tensors layer i uses."""
    while "weights_of" in config["layers"][i]:
        i = config["layers"][i]["weights_of"]
    return i


# ------------------------------------------------------------------------------------------- the model
def forward(tokens, config, weights, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  `layers_out`: a list that receives the residual after each layer."""
    eps, groups, alpha = config["norm"]["eps"], config["norm"]["groups"], config["postln_alpha"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{owner(config, i)}.")
        x = join(x, MIXERS[layer["type"]](x, _sub(w, "mix."), layer["mixer"], eps), w["norm1"], alpha, groups, eps)
        if layer["mlp"] is not None:
            x = join(x, feed_forward(x, _sub(w, "mlp.")), w["norm2"], alpha, groups, eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(grouped_norm(x, weights["final.norm"], groups, eps), weights["head"])


def greedy(prompt, n, config, weights):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(forward(toks, config, weights)[-1].argmax()))
    return toks[len(prompt):]


# ------------------------------------------------------------------------------------------- test models
def tensor_shapes(config):
    """Name -> shape of every tensor of a model."""
    W, V = config["width"], config["vocab"]
    out = {"embed": (V, W), "final.norm": (W,), "head": (V, W)}
    for i, layer in enumerate(config["layers"]):
        if "weights_of" in layer:
            continue
        p, m = f"l{i}.", layer["mixer"]
        x, H = p + "mix.", m["heads"]
        out[p + "norm1"] = (W,)
        if layer["type"] == "latent_attention":
            rank = m["kv_rank"]
            out.update({x + "q": (H * (m["dim"] + m["rot_dim"]), W), x + "dkv": (rank + m["rot_dim"], W), x + "dkv.norm": (rank,),
                        x + "uk": (H * m["dim"], rank), x + "uv": (H * m["vdim"], rank), x + "sink": (H,), x + "g": (H, W),
                        x + "o": (W, H * m["vdim"])})
        else:
            size = {"q": H * m["dim"], "k": m["kv_heads"] * m["dim"], "v": m["kv_heads"] * m["vdim"]}
            out.update({x + n: (s, W) for n, s in size.items()})
            out.update({x + n + ".conv": (s, m["conv"]) for n, s in size.items()})
            out.update({x + "q.norm": (size["q"],), x + "k.norm": (size["k"],), x + "talk": (H, H), x + "o": (W, H * m["vdim"])})
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
    return out


def random_weights(config, seed=0):
    """bfloat16 weights of a sensible scale: linear maps keep the variance, norms sit around one."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        r = torch.randn(shape, generator=g)
        if name.endswith(".conv"):
            t = r * 0.4
            t[:, -1] += 0.7
        elif name.endswith("sink"):
            t = 1.5 * r
        elif name.endswith("talk"):
            t = 0.6 * torch.eye(shape[0]) + 0.5 * r * shape[1] ** -0.5
        elif len(shape) == 1:
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = r * 0.7
        else:
            t = r * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
