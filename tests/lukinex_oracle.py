"""A plain, slow Lukinex: one function per mechanism, one head or one token at a time, whole sequences, no cache.

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


def linear(x, w, b=None):
    y = jitter(x) @ w.T
    return jitter(y if b is None else y + b)


# ------------------------------------------------------------------------------------------- mechanisms
def rms_norm(x, w, eps):
    """x over its root mean square along the last dimension (eps inside the root), times w."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def short_conv(x, w):
    """Causal convolution per channel: x [T, C], w [C, taps], the last column belongs to the current token."""
    y = torch.zeros_like(x)
    taps = w.shape[1]
    for back in range(taps):
        n = x.shape[0] - back
        if n > 0:
            y[back:] += x[:n] * w[:, taps - 1 - back]
    return y


def rotate(x, rot, first_position=0):
    """Rotary positions on the first `dims` of every head of x [T, heads, dim], i paired with i + dims/2; a linear
    scaling divides every frequency by its factor."""
    y = x.clone()
    dims = rot["dims"]
    half = dims // 2
    position = first_position + torch.arange(x.shape[0], dtype=torch.float64)
    for i in range(half):
        f = rot["base"] ** (-2.0 * i / dims)
        if rot.get("scaling"):
            f = f / rot["scaling"]["factor"]
        c, s = (position * f).cos().to(x.dtype)[:, None], (position * f).sin().to(x.dtype)[:, None]
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i] = u * c - v * s
        y[:, :, i + half] = v * c + u * s
    return y


def visible(T, window=None, keep=0):
    """[T, T]: may query i (row) see key j?  Inside the window (None: everything before it), or among the first `keep`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if window is None else i - j < window
    return (j <= i) & (near | (j < keep))


def attention(q, k, v, scale, mask, softcap=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: query head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = q.new_zeros(T, H, v.shape[-1])
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if softcap is not None:
            s = softcap * torch.tanh(s / softcap)
        s = s.masked_fill(~mask, -math.inf)
        p = torch.exp(s - s.max(-1, keepdim=True).values)
        out[:, h] = (p / p.sum(-1, keepdim=True)) @ v[:, g]
    return out


def lightning(q, k, v, decay):
    """Token by token from S = 0: S <- decay * S + k v^T, o = S^T q.  q, k [T, H, dk]; v [T, H, dv]; decay [H]."""
    T, H, dk = q.shape
    S = q.new_zeros(H, dk, v.shape[-1])
    a = torch.tensor(decay, dtype=q.dtype)[:, None, None]
    out = q.new_zeros(T, H, v.shape[-1])
    for t in range(T):
        S = a * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def clamped_glu(gate, up, limit):
    g = torch.clamp(gate, max=limit)
    u = torch.clamp(up, min=-limit, max=limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def route(z, top):
    """Router logits z [T, E] -> (expert ids [T, top], weights [T, top]): softmax over the chosen ones."""
    ids, ws = [], []
    for t in range(z.shape[0]):
        order = sorted(range(z.shape[1]), key=lambda e: -float(z[t, e]))[:top]
        e = torch.exp(z[t][order] - z[t][order].max())
        ids.append(order)
        ws.append(e / e.sum())
    return torch.tensor(ids), torch.stack(ws)


# ------------------------------------------------------------------------------------------- sublayers
def attention_mixer(h, w, cfg, eps, shared):
    T, H, G, d, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q = rms_norm(linear(h, w["q"]).view(T, H, d), w["q.norm"], eps)
    k = rms_norm(linear(h, w["k"]).view(T, G, d), w["k.norm"], eps)
    v = linear(h, w["v"]).view(T, G, dv)
    mask = visible(T, cfg["mask"]["size"], cfg["mask"]["keep_first"])
    o = attention(jitter(rotate(q, cfg["rot"])), jitter(rotate(k, cfg["rot"])), v, cfg["scale"], mask)
    return linear(o.reshape(T, H * dv), w["o"])


def convolved_attention(h, w, cfg):
    T, H, G, d, dv = h.shape[0], cfg["heads"], cfg["kv_heads"], cfg["dim"], cfg["vdim"]
    q, k, v = (short_conv(linear(h, w[n], w[n + ".b"]), w[n + ".conv"]) for n in "qkv")
    q, k = rotate(q.view(T, H, d), cfg["rot"]), rotate(k.view(T, G, d), cfg["rot"])
    mask = visible(T, cfg["mask"]["size"], cfg["mask"]["keep_first"])
    o = attention(jitter(q), jitter(k), jitter(v.view(T, G, dv)), cfg["scale"], mask, cfg["softcap"])
    return linear(o.reshape(T, H * dv), w["o"], w["o.b"])


def lightning_mixer(h, w, cfg, eps):
    T, H, dk, dv = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"]
    q, k = (silu(linear(h, w[n])).view(T, H, dk) for n in "qk")
    v = silu(linear(h, w["v"])).view(T, H, dv)
    o = rms_norm(lightning(q, k, jitter(v), cfg["decay"]).reshape(T, H * dv), w["norm"], eps)
    return linear(o * sigmoid(linear(h, w["g"])), w["o"])


def parallel_mixer(h, w, cfg, eps, shared):
    left = convolved_attention(h, _sub(w, "left."), cfg["left"])
    right = lightning_mixer(h, _sub(w, "right."), cfg["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def latent_mixer(h, w, cfg, eps, shared):
    """`shared`: layer index -> its latents; a layer with `kv_from` reads another's."""
    T, H, d, dv, r = h.shape[0], cfg["heads"], cfg["dim"], cfg["vdim"], cfg["kv_rank"]
    q = linear(rms_norm(linear(h, w["dq"]), w["dq.norm"], eps), w["uq"]).view(T, H, d)
    if "kv_from" in cfg:
        c = shared[cfg["kv_from"]]
    else:
        c = shared["own"] = rms_norm(linear(h, w["dkv"]), w["dkv.norm"], eps)
    k, v = linear(c, w["uk"]).view(T, H, d), linear(c, w["uv"]).view(T, H, dv)
    return linear(attention(q, k, v, cfg["scale"], visible(T)).reshape(T, H * dv), w["o"])


def expert(h, w, limit):
    return linear(clamped_glu(linear(h, w["gate"]), linear(h, w["up"]), limit), w["down"])


def experts(h, w, cfg):
    ids, weights = route(h @ w["router"].T, cfg["router"]["top"])
    out = expert(h, _sub(w, "shared."), cfg["shared"]["limit"])
    for e in range(cfg["router"]["experts"]):
        picked = (ids == e).nonzero()
        if len(picked):
            y = expert(h, _sub(w, f"e{e}."), cfg["expert"]["limit"])
            for t, j in picked.tolist():
                out[t] += weights[t, j] * y[t]
    return out


MIXERS = {"attention": attention_mixer, "parallel": parallel_mixer, "latent_attention": latent_mixer}


def _sub(w, prefix):
    return {n[len(prefix):]: t for n, t in w.items() if n.startswith(prefix)}


# ------------------------------------------------------------------------------------------- the model
def forward(tokens, config, weights, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  `layers_out`: a list that receives the residual after each layer."""
    eps = config["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    shared = {}
    for i, layer in enumerate(config["layers"]):
        w = _sub(weights, f"l{i}.")
        y = MIXERS[layer["type"]](rms_norm(x, w["norm1"], eps), _sub(w, "mix."), layer["mixer"], eps, shared)
        if "own" in shared:
            shared[i] = shared.pop("own")
        x = x + rms_norm(y, w["norm1b"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(experts(rms_norm(x, w["norm2"], eps), _sub(w, "mlp."), layer["mlp"]), w["norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x)
    return linear(rms_norm(x, weights["final.norm"], eps), weights["head"])


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
        p, m = f"l{i}.", layer["mixer"]
        x = p + "mix."
        out.update({p + "norm1": (W,), p + "norm1b": (W,)})
        if layer["type"] == "latent_attention":
            H, r = m["heads"], m["kv_rank"]
            out.update({x + "dq": (m["q_rank"], W), x + "dq.norm": (m["q_rank"],), x + "uq": (H * m["dim"], m["q_rank"]),
                        x + "uk": (H * m["dim"], r), x + "uv": (H * m["vdim"], r), x + "o": (W, H * m["vdim"])})
            if "kv_from" not in m:
                out.update({x + "dkv": (r, W), x + "dkv.norm": (r,)})
        else:
            a, at = (m, x) if layer["type"] == "attention" else (m["left"], x + "left.")
            size = {"q": a["heads"] * a["dim"], "k": a["kv_heads"] * a["dim"], "v": a["kv_heads"] * a["vdim"]}
            out.update({at + n: (s, W) for n, s in size.items()})
            out[at + "o"] = (W, a["heads"] * a["vdim"])
            if layer["type"] == "attention":
                out.update({at + "q.norm": (a["dim"],), at + "k.norm": (a["dim"],)})
            else:
                out.update({at + n + ".b": (s,) for n, s in size.items()})
                out.update({at + n + ".conv": (s, a["conv"]) for n, s in size.items()})
                r, at = m["right"], x + "right."
                out.update({x + "left.o.b": (W,), at + "q": (r["heads"] * r["dim"], W), at + "k": (r["heads"] * r["dim"], W),
                            at + "v": (r["heads"] * r["vdim"], W), at + "g": (r["heads"] * r["vdim"], W),
                            at + "o": (W, r["heads"] * r["vdim"]), at + "norm": (r["heads"] * r["vdim"],),
                            x + "left.out": (W,), x + "right.out": (W,)})
        if layer["mlp"] is not None:
            f, q = layer["mlp"], p + "mlp."
            E = f["router"]["experts"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), q + "router": (E, W)})
            for n, ff in [(f"{q}e{e}.", f["expert"]["ff"]) for e in range(E)] + [(q + "shared.", f["shared"]["ff"])]:
                out.update({n + "gate": (ff, W), n + "up": (ff, W), n + "down": (W, ff)})
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
        elif name.endswith(".b"):
            t = 0.3 * r
        elif len(shape) == 1:
            t = 1.0 + 0.2 * r
        elif name == "embed":
            t = r * 0.7
        elif name.endswith("router"):
            t = 2.0 * r * shape[1] ** -0.5
        else:
            t = r * shape[1] ** -0.5
        out[name] = t.to(torch.bfloat16)
    return out
