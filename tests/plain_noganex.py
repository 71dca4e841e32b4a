"""A plain, slow restatement of the Noganex design, written from its equations: one function per mechanism, whole
sequences, float64, no cache, no kernels, nothing shared with the package.  The GPU tests hold the engine to it.

Notation: T tokens, W the model's width, x the residual stream [T, W], positions p = 0..T-1, n(v; w) the RMS norm
v / sqrt(mean(v^2) + eps) * w.

  embedding      x = E[token]
  layer          x <- x + n(mixer(x) * sigmoid(R1 x + r1); norm1);  x <- x + n(ff(x) * sigmoid(R2 x + r2); norm2)
  attention      q = rot(n(Wq x; over all heads' lanes at once)), k likewise, v = Wv x;  s_h = scale * q_h . k_kv(h);
                 s'_h = sum_g talk[h, g] s_g;  softmax of s' over the keys of the query's own chunk, up to itself;  Wo
  rotation       lane i with lane i + dims/2 of the first dims lanes, angle p f_i, frequencies slowed by a ramp over i
  delta          q, k, v = silu(conv(W x));  q, k unit vectors, q / sqrt(dim);  b = sigmoid(Wb x);
                 g = exp(-exp(A) softplus(Wa x + dt));  S <- g S;  u = b (v - S^T k);  S <- S + k u^T;  o = S^T q;
                 o <- n(o; per head) * silu(Wg x);  Wo
  dense          Wd (gelu_tanh(Wg x + bg) * (Wu x + bu)) + bd
  experts        s = sigmoid(Wr x);  chosen = top(s + correction);  a_e = scale * s_e / (sum of the chosen s + 1e-20);
                 sum_e a_e E_e(x) + shared(x);  E(x) = Wd (silu(Wg x) * (Wu x))
  head           logits = (H n(x; final)) * logit_scale
A layer with ``weights_of`` runs the tensors of another layer on a state of its own.
"""

import math

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- mechanisms


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def gated_normed(y, gate, w, eps):
    """What a sublayer adds to the stream: its output times the logistic function of the gate's logits, then normed."""
    return rms_norm(y * torch.sigmoid(gate), w, eps)


def ramp_frequencies(dims, base, scaling=None):
    """(frequencies [dims / 2], factor of cos and sin)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
    index = lambda turns: dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(index(fast)), 0), min(math.ceil(index(slow)), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / factor * r + v * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate_half(x, dims, base, scaling=None, first=0):
    """x [T, heads, d] at positions first..first+T-1: lane i turns with lane i + dims/2, the lanes from dims on stay.  The
    design takes angles in 32 bits: the frequency is rounded to a float, and so is its product with the position."""
    f, factor = ramp_frequencies(dims, base, scaling)
    pos = torch.arange(first, first + x.shape[0], dtype=torch.float32)
    a = (pos[:, None] * torch.tensor(f, dtype=F64).float()[None]).to(F64)
    cos, sin = (torch.cos(a) * factor)[:, None], (torch.sin(a) * factor)[:, None]
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def same_chunk(T, size=None):
    """[T, T] booleans: row p sees column j."""
    p = torch.arange(T)
    seen = p[None, :] <= p[:, None]
    return seen if size is None else seen & (p[None, :] // size == p[:, None] // size)


def mixed_attend(q, k, v, scale, talk, seen):
    """q [T, H, d], k [J, G, d], v [J, G, dv], talk [H, H] or None, seen [T, J] -> [T, H, dv]."""
    rep = q.shape[1] // k.shape[1]
    s = torch.einsum("phd,jhd->hpj", q, k.repeat_interleave(rep, 1)) * scale
    if talk is not None:
        s = torch.einsum("hg,gpj->hpj", talk, s)
    s = s.masked_fill(~seen[None], float("-inf"))
    return torch.einsum("hpj,jhd->phd", torch.softmax(s, -1), v.repeat_interleave(rep, 1))


def attention(w, p, m, h, eps):
    T, H, G = h.shape[0], m["heads"], m.get("kv_heads", m["heads"])
    d, dv = m["dim"], m.get("vdim", m["dim"])
    q = rms_norm(h @ w[p + "q"].T, w[p + "q.norm"], eps).view(T, H, d)
    k = rms_norm(h @ w[p + "k"].T, w[p + "k.norm"], eps).view(T, G, d)
    v = (h @ w[p + "v"].T).view(T, G, dv)
    rot = m.get("rot")
    if rot:
        q, k = (rotate_half(x, rot["dims"], rot["base"], rot.get("scaling")) for x in (q, k))
    out = mixed_attend(q, k, v, m["scale"], w[p + "talk"], same_chunk(T, (m.get("mask") or {}).get("size")))
    return out.reshape(T, H * dv) @ w[p + "o"].T


def causal_convolution(x, taps):
    """x [T, C], taps [C, n] (the last column weighs the current token), zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x], 0)
    return sum(padded[j:j + T] * taps[:, j] for j in range(n))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, beta, decay):
    """q, k [T, H, d], v [T, H, dv], beta, decay [T, H] -> the read-outs [T, H, dv] and the last state [H, d, dv]."""
    T, H, d = k.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64)
    out = torch.zeros_like(v)
    for t in range(T):
        S = S * decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - torch.einsum("hij,hi->hj", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return out, S


def delta_core(m, qkv, b, a, gate, taps, A_log, dt_bias, norm, eps):
    """The mixer between its projections: qkv [T, channels] before the convolutions, b, a [T, heads], gate
    [T, heads * vdim] -> [T, heads * vdim]."""
    T, H, G = qkv.shape[0], m["heads"], m.get("kv_heads", m["heads"])
    d, dv = m["dim"], m["vdim"]
    y = silu(causal_convolution(qkv, taps))
    q = unit(y[:, :G * d].view(T, G, d)).repeat_interleave(H // G, 1) / math.sqrt(d)
    k = unit(y[:, G * d:2 * G * d].view(T, G, d)).repeat_interleave(H // G, 1)
    v = y[:, 2 * G * d:].view(T, H, dv)
    decay = torch.exp(-torch.exp(A_log) * torch.nn.functional.softplus(a + dt_bias))
    o, _ = delta_recurrence(q, k, v, torch.sigmoid(b), decay)
    return rms_norm(o, norm, eps).reshape(T, H * dv) * silu(gate)


def delta(w, p, m, h, eps):
    qkv = torch.cat([h @ w[p + r].T for r in ("q", "k", "v")], -1)
    taps = torch.cat([w[p + r + ".conv"] for r in ("q", "k", "v")], 0)
    out = delta_core(m, qkv, h @ w[p + "b"].T, h @ w[p + "a"].T, h @ w[p + "g"].T, taps, w[p + "A_log"], w[p + "dt_bias"],
                     w[p + "norm"], eps)
    return out @ w[p + "o"].T


def dense_feed_forward(w, p, h):
    g = h @ w[p + "gate"].T + w[p + "gate.b"]
    u = h @ w[p + "up"].T + w[p + "up.b"]
    return (gelu_tanh(g) * u) @ w[p + "down"].T + w[p + "down.b"]


def silu_expert(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def router_choice(logits, correction, top, scale):
    """(indices [T, top] by falling choice score, the lower index first among equals; weights [T, top])."""
    s = torch.sigmoid(logits)
    chosen = torch.sort(s + correction, dim=-1, descending=True, stable=True).indices[:, :top]
    picked = torch.gather(s, 1, chosen)
    return chosen, picked / (picked.sum(-1, keepdim=True) + 1e-20) * scale


def routed_feed_forward(w, p, f, h):
    r = f["router"]
    chosen, weights = router_choice(h @ w[p + "router"].T, w[p + "correction"], r["top"], r.get("scale", 1.0))
    out = torch.zeros(h.shape[0], w[p + "e0.down"].shape[0], dtype=F64)
    for e in range(r["experts"]):
        share = (weights * (chosen == e)).sum(-1)
        rows = share.nonzero().flatten()
        if len(rows):
            out[rows] += share[rows, None] * silu_expert(w, f"{p}e{e}.", h[rows])
    if f.get("shared"):
        out = out + silu_expert(w, p + "shared.", h)
    return out


def owner(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, weights, tokens, keep_layers=False):
    """Logits [T, vocab] of the whole sequence (and, with ``keep_layers``, the stream after every layer)."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.tensor(tokens)]
    streams = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, i)}."
        mixer = attention if layer["type"] == "attention" else delta
        y = mixer(w, p + "mix.", layer["mixer"], x, eps)
        x = x + gated_normed(y, x @ w[p + "rg1"].T + w[p + "rg1.b"], w[p + "norm1"], eps)
        f = layer.get("mlp")
        if f is not None:
            y = dense_feed_forward(w, p + "mlp.", x) if f["kind"] == "dense" else routed_feed_forward(w, p + "mlp.", f, x)
            x = x + gated_normed(y, x @ w[p + "rg2"].T + w[p + "rg2.b"], w[p + "norm2"], eps)
        streams.append(x.clone())
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T * cfg.get("logit_scale", 1.0)
    return (logits, torch.stack(streams)) if keep_layers else logits


# ----------------------------------------------------------------------------- configurations and weights


def _attention(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None, base=10000.0, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot:
        m["rot"] = {"base": base, "dims": rot}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return {"type": "attention", "mixer": m}


def _delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def _dense(ff):
    return {"kind": "dense", "ff": ff}


def _moe(experts, top, ff, scale=1.0, shared=None):
    f = {"kind": "moe", "router": {"experts": experts, "top": top, "scale": scale}, "expert": {"ff": ff}}
    if shared:
        f["shared"] = {"ff": shared}
    return f


def _config(vocab, width, layers, logit_scale=1.0, eps=1e-5):
    return {"architecture": "Noganex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [{**mixer, "mlp": mlp, **({} if of is None else {"weights_of": of})} for mixer, mlp, of in layers]}


# every size differs from its neighbours; three query heads a key head; a chunk off the page size; a shared layer of each kind
_A0, _A1 = _attention(6, 2, 32, 24, 0.21, 40, 20, 5000.0, (4.0, 512, 16.0, 2.0)), _delta(6, 3, 24, 40, 4)
TINY_A = _config(150, 104, [(_A0, _moe(6, 2, 40, 1.7, 24), None), (_A1, _dense(72), None), (_A0, _moe(6, 2, 40, 1.7, 24), 0),
                            (_A1, _dense(72), 1), (_delta(2, 2, 16, 16, 2), None, None)], 0.7)
# sizes off the multiples of 8 and 16: the kernels' general forms; no chunk, no slowed frequencies, one expert a token
TINY_B = _config(97, 90, [(_delta(3, 1, 10, 7, 1), _moe(5, 1, 28, 0.5), None),
                          (_attention(3, 3, 20, 12, 0.3, None, 10), _dense(50), None),
                          (_attention(4, 1, 18, 30, 0.25, 33, 18, 700.0), None, None)], 1.9, 1e-6)
# chunks of one page, of less and of more than one, and a delta mixer that a layer before its owner borrows
_C3 = _delta(4, 4, 32, 16, 5)
TINY_C = _config(120, 64, [(_attention(4, 2, 16, 32, 0.25, 64, 16), _dense(48), None), (_C3, _moe(4, 3, 32, 2.0, 16), 3),
                           (_attention(8, 4, 16, 16, 0.25, 130, 8, 10000.0, (2.0, 64, 4.0, 1.0)), _dense(40), None),
                           (_C3, _moe(4, 3, 32, 2.0, 16), None)], 0.3)
# heads of 96, 80, 64 and 128 lanes, which take other kernel forms than the small ones
TINY_D = _config(200, 160, [(_attention(5, 5, 96, 80, 0.1, 100, 96), _moe(7, 4, 64, 2.5, 32), None),
                            (_delta(4, 2, 64, 128, 4), _dense(200), None),
                            (_attention(4, 2, 128, 128, 0.09, 90, 64), _dense(64), None),
                            (_delta(2, 1, 128, 64, 3), _moe(3, 2, 48, 1.2), None)], 1.3)
# sharpened softmaxes with chunks of hundreds of positions
SHARP = _config(90, 64, [(_attention(4, 2, 16, 16, 0.5, 200, 16), None, None),
                         (_attention(4, 4, 16, 16, 0.5, 300, 8), _dense(48), None), (_delta(4, 2, 16, 16, 3), None, None)])


def tensor_shapes(cfg):
    """Name -> shape of every tensor that a model of this configuration stores."""
    W, V = cfg["width"], cfg["vocab"]
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        if layer.get("weights_of") is not None:
            continue
        p, m = f"l{i}.", layer["mixer"]
        H, G, d, dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m.get("vdim", m["dim"])
        shapes.update({p + "norm1": (W,), p + "rg1": (W, W), p + "rg1.b": (W,), p + "mix.q": ((H if layer["type"] == "attention" else G) * d, W),
                       p + "mix.k": (G * d, W), p + "mix.o": (W, H * dv)})
        if layer["type"] == "attention":
            shapes.update({p + "mix.v": (G * dv, W), p + "mix.q.norm": (H * d,), p + "mix.k.norm": (G * d,), p + "mix.talk": (H, H)})
        else:
            shapes.update({p + "mix.v": (H * dv, W), p + "mix.g": (H * dv, W), p + "mix.a": (H, W), p + "mix.b": (H, W),
                           p + "mix.A_log": (H,), p + "mix.dt_bias": (H,), p + "mix.norm": (dv,)})
            for r, n in (("q", G * d), ("k", G * d), ("v", H * dv)):
                shapes[f"{p}mix.{r}.conv"] = (n, m["conv"])
        f = layer.get("mlp")
        if f is None:
            continue
        shapes.update({p + "norm2": (W,), p + "rg2": (W, W), p + "rg2.b": (W,)})
        if f["kind"] == "dense":
            F = f["ff"]
            shapes.update({p + "mlp.gate": (F, W), p + "mlp.gate.b": (F,), p + "mlp.up": (F, W), p + "mlp.up.b": (F,),
                           p + "mlp.down": (W, F), p + "mlp.down.b": (W,)})
        else:
            n = f["router"]["experts"]
            shapes.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
            blocks = [(f"e{e}.", f["expert"]["ff"]) for e in range(n)]
            if f.get("shared"):
                blocks.append(("shared.", f["shared"]["ff"]))
            for name, F in blocks:
                shapes.update({f"{p}mlp.{name}gate": (F, W), f"{p}mlp.{name}up": (F, W), f"{p}mlp.{name}down": (W, F)})
    return shapes


def random_weights(cfg, seed, sharpen=1.0):
    """Every tensor of the design, rounded to bfloat16 values so that both compute dtypes hold the same numbers."""
    gen = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        z = torch.randn(shape, generator=gen)
        last = name.rsplit(".", 1)[-1]
        if name == "embed":
            pass
        elif last == "talk":
            z = torch.eye(shape[0]) + 0.4 * z          # not symmetric, off-diagonal entries that matter
        elif last == "conv":
            z = 0.3 * z
            z[:, -1] += 0.8
        elif last == "A_log":
            z = torch.log(0.03 + 0.5 * torch.rand(shape, generator=gen))      # memory over tens of tokens
        elif last == "dt_bias":
            z = 0.5 * z - 1.0
        elif last == "correction":
            z = 0.15 * z
        elif last == "b":
            z = 0.3 * z if len(shape) == 1 else z / math.sqrt(shape[1])
        elif len(shape) == 1:
            z = 1.0 + 0.15 * z
            if name.endswith("mix.q.norm"):
                z = z * sharpen
        else:
            gain = {"router": 2.0, "gate": 1.5, "up": 1.5}.get(last, 1.0)
            z = z * gain / math.sqrt(shape[-1])
        out[name] = z
    for name in list(out):
        if name.endswith(("norm1", "norm2")):
            out[name] = 0.6 * out[name]
    return {k: v.to(torch.bfloat16) for k, v in out.items()}


def random_prompts(cfg, lengths, seed):
    gen = torch.Generator().manual_seed(1000 + seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=gen).tolist() for n in lengths]


def random_config(seed):
    """A configuration drawn from odd sizes: widths off the multiples of 8, head counts that do not divide alike, chunks
    beside the page size, with and without each optional mechanism, layers that borrow the tensors of others."""
    gen = torch.Generator().manual_seed(8000 + seed)
    pick = lambda *values: values[int(torch.randint(0, len(values), (1,), generator=gen))]
    layers = []
    for i in range(pick(2, 3, 4)):
        of = int(pick(*range(i))) if i and pick(0, 0, 1) else None
        if of is not None:
            while layers[of][2] is not None:
                of = layers[of][2]
            layers.append((layers[of][0], layers[of][1], of))
            continue
        kv = pick(1, 2, 3)
        heads = kv * pick(1, 2, 4)
        if pick(0, 1):
            dim = pick(6, 16, 20, 48)
            rot = pick(*[r for r in (2, 6, 16, 20, 48) if r <= dim])
            mixer = _attention(heads, kv, dim, pick(5, 16, 40), pick(0.1, 0.3), pick(None, 1, 17, 48, 64, 90, 128), rot,
                               pick(300.0, 10000.0), pick(None, (2.0, 256, 32.0, 1.0), (8.0, 64, 3.0, 0.5)))
        else:
            mixer = _delta(heads, kv, pick(6, 16, 33, 48), pick(5, 16, 40), pick(1, 2, 4))
        f = pick(None, "dense", "moe", "moe")
        if f == "dense":
            f = _dense(pick(10, 24, 52))
        elif f == "moe":
            experts = pick(2, 3, 7)
            f = _moe(experts, pick(*range(1, experts + 1)), pick(6, 16, 28), pick(1.0, 2.5), pick(None, 12))
        layers.append((mixer, f, None))
    return _config(pick(50, 131), pick(36, 50, 64, 72), layers, pick(1.0, 0.25, 3.0), pick(1e-5, 1e-6))
