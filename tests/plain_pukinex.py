"""A plain, slow restatement of the Pukinex design, written from its equations: one function per mechanism, whole
sequences, float64, no cache, no kernels, nothing shared with the package.  The GPU tests hold the engine to it.

Notation: T tokens, W the model's width, S parallel streams X [S, T, W], positions p = 0..T-1, ln(v) the layer norm
(v - mean) / sqrt(var + eps) * w + b, rms(v) = v / sqrt(mean(v^2) + eps), sg the logistic function.

  embedding   X_s = E[token] * c                                             for every stream s
  sublayer    u = sum_s in_s X_s;  y = f(ln(u));  X_t <- sum_s mix[s, t] X_s + m out_t y       (f: mixer, then feed-forward)
  attention   q = Wq h, k = Wk h, v = k;  q, k rotated (neighbouring lanes, slowed by a factor);
              s = c tanh(scale q . k / c);  p_j = e^(s_j) / (1 + sum e^(s_k));  o_h * sg(Wg h)_h;  Wo
  parallel    a * left(h) + b * right(h)
    left      q, k, v with biases;  q, k <- rms * weight per head;  q *= 1 + coef ln(floor((p + 1) / every) + 1);
              s = scale q . k + rel[bucket(p - j), head];  p_j as above;  o * sg(Wg h) lane by lane;  Wo
    right     q, k rotated (lane i with lane i + dims/2), k * dim^(-1/2);  S <- decay S + k v^T;  o = S^T q;
              rms(o) per head * silu(Wg h);  Wo
  dense       Wd max(Wu h, 0)^2
  head        x = sum_s X_s;  z = (H ln(x)) * logit_scale;  logits = c tanh(z / c)
A looped range of layers runs several times in a row with the same tensors.
"""

import math

import torch

F64 = torch.float64


# ----------------------------------------------------------------------------- mechanisms


def layer_norm(x, w, b, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * w + b


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def stream_input(X, weights):
    """X [S, T, W], weights [S] -> what a sublayer's norm reads."""
    return sum(weights[s] * X[s] for s in range(X.shape[0]))


def stream_update(X, mix, out, m, y):
    """The new streams, all from the old ones: mix[s, t] leads from stream s to stream t."""
    S = X.shape[0]
    return torch.stack([sum(mix[s, t] * X[s] for s in range(S)) + m * out[t] * y for t in range(S)])


def angles(positions, dims, base, factor=1.0):
    """[T, dims / 2]: taken in 32 bits, as the design does (a rounded frequency times the position, rounded)."""
    f = torch.tensor([base ** (-2.0 * i / dims) / factor for i in range(dims // 2)], dtype=F64).float()
    return (positions.float()[:, None] * f[None]).to(F64)


def rotate(x, dims, base, factor=1.0, neighbours=True, first=0):
    """x [T, heads, d] at positions first.. : the first ``dims`` lanes turn in pairs of neighbours, or of halves."""
    a = angles(torch.arange(first, first + x.shape[0]), dims, base, factor)
    cos, sin = torch.cos(a)[:, None], torch.sin(a)[:, None]
    out = x.clone()
    if neighbours:
        u, v = x[..., 0:dims:2], x[..., 1:dims:2]
        out[..., 0:dims:2], out[..., 1:dims:2] = u * cos - v * sin, v * cos + u * sin
    else:
        u, v = x[..., :dims // 2], x[..., dims // 2:dims]
        out[..., :dims // 2], out[..., dims // 2:dims] = u * cos - v * sin, v * cos + u * sin
    return out


def temperature(positions, coef, every):
    return torch.tensor([1.0 + coef * math.log((int(p) + 1) // every + 1) for p in positions], dtype=F64)


def bucket(n, rows, reach):
    """The row of a distance table that a distance of n positions reads: one row each for the near half, then rows
    whose widths grow, the last one for everything from about ``reach`` on."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half)))


def distance_bias(rel, queries, keys, reach):
    """[heads, P, J] of rel[bucket(p - j), head] (that of distance 0 where j > p, which nobody sees)."""
    distance = (torch.tensor(list(queries))[:, None] - torch.tensor(list(keys))[None]).clamp(min=0)
    rows = torch.tensor([bucket(n, rel.shape[0], reach) for n in range(int(distance.max()) + 1)])
    return rel[rows[distance]].permute(2, 0, 1)


def sink_attend(q, k, v, scale, softcap=None, bias=None):
    """q [P, H, d] at the last P positions of k [J, G, d], v [J, G, dv] -> [P, H, dv].  bias [H, P, J]."""
    P, J, rep = q.shape[0], k.shape[0], q.shape[1] // k.shape[1]
    s = torch.einsum("phd,jhd->hpj", q, k.repeat_interleave(rep, 1)) * scale
    if softcap is not None:
        s = softcap * torch.tanh(s / softcap)
    if bias is not None:
        s = s + bias
    seen = torch.arange(J)[None] <= torch.arange(J - P, J)[:, None]
    s = torch.cat([torch.zeros(s.shape[0], P, 1, dtype=s.dtype), s.masked_fill(~seen[None], float("-inf"))], -1)
    weights = torch.softmax(s, -1)[..., 1:]          # the first column: a score of 0 without a value
    return torch.einsum("hpj,jhd->phd", weights, v.repeat_interleave(rep, 1))


def attention(w, p, m, h):
    T, H, G, d = h.shape[0], m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    q, k = (h @ w[p + "q"].T).view(T, H, d), (h @ w[p + "k"].T).view(T, G, d)
    v = k
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        q, k = (rotate(x, rot["dims"], rot["base"], factor) for x in (q, k))
    out = sink_attend(q, k, v, m["scale"], m.get("softcap"))
    return (out * torch.sigmoid(h @ w[p + "g"].T)[:, :, None]).reshape(T, H * d) @ w[p + "o"].T


def left_heads(w, p, m, h, eps):
    """Queries, keys and values of the biased attention, ready for the scores."""
    T, H, G, d = h.shape[0], m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
    project = lambda r, heads: (h @ w[p + r].T + w[p + r + ".b"]).view(T, heads, -1)
    q = rms(project("q", H), eps) * w[p + "q.norm"]
    k = rms(project("k", G), eps) * w[p + "k.norm"]
    warm = m.get("q_temp")
    if warm:
        q = q * temperature(range(T), warm["coef"], warm["every"])[:, None, None]
    return q, k, project("v", G)


def left(w, p, m, h, eps):
    T = h.shape[0]
    q, k, v = left_heads(w, p, m, h, eps)
    out = sink_attend(q, k, v, m["scale"], bias=distance_bias(w[p + "rel"], range(T), range(T), m["bias_max"]))
    return (out.reshape(T, -1) * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def retention_recurrence(q, k, v, decay, S=None):
    """q, k [T, H, d], v [T, H, dv], decay [H] -> the read-outs [T, H, dv] and the last state [H, d, dv]."""
    S = torch.zeros(k.shape[1], k.shape[2], v.shape[2], dtype=q.dtype) if S is None else S
    out = torch.zeros_like(v)
    for t in range(q.shape[0]):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hij,hi->hj", S, q[t])
    return out, S


def retention_core(m, q, k, v, gate, eps, first=0, S=None):
    """The mixer between its projections: q, k [T, H d], v, gate [T, H dv] -> ([T, H dv], the last state)."""
    T, H, d, dv = q.shape[0], m["heads"], m["dim"], m.get("vdim", m["dim"])
    q, k = q.view(T, H, d), k.view(T, H, d)
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {}).get("factor", 1.0)
        q, k = (rotate(x, rot["dims"], rot["base"], factor, neighbours=False, first=first) for x in (q, k))
    out, S = retention_recurrence(q, k * d ** -0.5, v.view(T, H, dv), torch.tensor(m["decay"], dtype=F64), S)
    return rms(out, eps).reshape(T, H * dv) * silu(gate), S


def right(w, p, m, h, eps):
    out, _ = retention_core(m, *(h @ w[p + r].T for r in ("q", "k", "v", "g")), eps)
    return out @ w[p + "o"].T


def parallel(w, p, m, h, eps):
    return (m.get("left_scale", 1.0) * left(w, p + "left.", m["left"], h, eps)
            + m.get("right_scale", 1.0) * right(w, p + "right.", m["right"], h, eps))


def feed_forward(w, p, h):
    return torch.clamp(h @ w[p + "up"].T, min=0.0) ** 2 @ w[p + "down"].T


def layer_runs(cfg):
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return list(range(n))
    inner = list(range(loop["start"], loop["stop"]))
    return list(range(loop["start"])) + inner * loop["times"] + list(range(loop["stop"], n))


def forward(cfg, weights, tokens, keep_layers=False):
    """Logits [T, vocab] of the whole sequence (and, with ``keep_layers``, the sum of the streams after every layer)."""
    w = {k: v.to(F64) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    norm = lambda name, x: layer_norm(x, w[name], w[name + ".b"], eps)
    S = cfg.get("streams")
    x = w["embed"][torch.tensor(tokens)] * (cfg.get("embedding") or {}).get("scale", 1.0)
    X = x[None].repeat(S or 1, 1, 1)
    sums = []
    for i in layer_runs(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        mixer = (lambda h: attention(w, p + "mix.", layer["mixer"], h)) if layer["type"] == "attention" else \
            (lambda h: parallel(w, p + "mix.", layer["mixer"], h, eps))
        subs = [("1", mixer)] + ([("2", lambda h: feed_forward(w, p + "mlp.", h))] if layer.get("mlp") else [])
        for n, f in subs:
            if S:
                y = f(norm(p + "norm" + n, stream_input(X, w[f"{p}hc{n}.in"])))
                X = stream_update(X, w[f"{p}hc{n}.mix"], w[f"{p}hc{n}.out"], m, y)
            else:
                X = X + m * f(norm(p + "norm" + n, X[0]))
        sums.append(X.sum(0))
    logits = norm("final.norm", X.sum(0)) @ w["head"].T * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return (logits, torch.stack(sums)) if keep_layers else logits


# ----------------------------------------------------------------------------- configurations and weights


def _rot(base, dims, factor=None):
    return {"base": base, "dims": dims, **({} if factor is None else {"scaling": {"factor": factor}})}


def _attention(heads, kv_heads, dim, scale, softcap=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if softcap:
        m["softcap"] = softcap
    if rot:
        m["rot"] = rot
    return {"type": "attention", "mixer": m}


def _left(heads, kv_heads, dim, vdim, scale, rows, reach, temp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "bias_rows": rows, "bias_max": reach}
    if temp:
        m["q_temp"] = dict(zip(("coef", "every"), temp))
    return m


def _right(decay, dim, vdim, rot=None):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay), **({"rot": rot} if rot else {})}


def _parallel(left, right, a=1.0, b=1.0):
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": a, "right_scale": b}}


def _config(vocab, width, layers, streams=None, loop=None, scale=1.0, m=1.0, logit_scale=1.0, cap=None, eps=1e-5):
    cfg = {"architecture": "Pukinex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
           "residual_mult": m, "logit_scale": logit_scale,
           "layers": [{**mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for mixer, ff in layers]}
    if streams:
        cfg["streams"] = streams
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if cap:
        cfg["logit_softcap"] = cap
    return cfg


# every size differs from its neighbours; a loop over two layers; a layer without a feed-forward
TINY_A = _config(150, 104, [
    (_parallel(_left(6, 2, 32, 24, 0.21, 12, 40, (0.4, 16)), _right((0.9, 0.995, 0.5), 24, 40, _rot(5000.0, 16)), 1.3, 0.6), 72),
    (_attention(4, 2, 32, 0.2, 20.0, _rot(3000.0, 20, 4.0)), 56),
    (_parallel(_left(4, 4, 16, 48, 0.3, 10, 70, (0.2, 10)), _right((0.97, 0.8), 16, 32, _rot(1e6, 16)), 0.7, 1.2), None)],
    streams=2, loop=(1, 3, 2), scale=3.0, m=0.6, logit_scale=0.7, cap=15.0)
# sizes off the multiples of 8 and 16: the kernels' general forms; an odd table, no cap, no slowed frequencies, no temperature
TINY_B = _config(97, 90, [
    (_parallel(_left(3, 3, 20, 12, 0.3, 7, 33), _right((0.9, 1.0), 10, 7, _rot(700.0, 6)), 0.9, 0.4), 50),
    (_attention(3, 1, 18, 0.25, None, _rot(400.0, 18)), 28),
    (_parallel(_left(5, 1, 18, 30, 0.2, 2, 9, (0.5, 7)), _right((0.7,), 33, 5), 1.0, 1.0), 10)],
    streams=3, scale=2.0, logit_scale=1.9, eps=1e-6)
# one plain stream, heads of 64 lanes, nothing optional
TINY_C = _config(120, 64, [(_attention(4, 2, 64, 0.12), 48), (_parallel(_left(4, 2, 64, 64, 0.13, 16, 100), _right((0.98, 0.9), 40, 96)), 40),
                           (_attention(2, 2, 64, 0.1, 10.0, _rot(10000.0, 32, 2.0)), None)])
# heads of 128, 96 and 80 lanes, six streams, a loop over everything
TINY_D = _config(200, 160, [
    (_parallel(_left(5, 5, 96, 80, 0.1, 20, 64, (0.3, 32)), _right((0.99, 0.93), 64, 128, _rot(1e4, 64)), 1.1, 0.8), 200),
    (_attention(4, 2, 128, 0.09, 30.0, _rot(1e4, 64, 8.0)), 64),
    (_parallel(_left(4, 2, 128, 128, 0.09, 32, 150, (0.3, 50)), _right((0.96,), 128, 64, _rot(1e4, 32)), 1.0, 1.0), None)],
    streams=6, loop=(0, 3, 2), scale=2.0, m=0.7, cap=20.0)
# sharpened softmaxes that pick keys anywhere in hundreds of positions, and a slow decay
SHARP = _config(90, 64, [(_parallel(_left(4, 2, 16, 16, 0.5, 16, 300, (0.3, 64)), _right((0.998, 0.99), 16, 16, _rot(1e4, 16))), None),
                         (_attention(4, 4, 16, 0.5, 40.0, _rot(1e4, 8, 3.0)), 48)], streams=2)


def tensor_shapes(cfg):
    """Name -> shape of every tensor that a model of this configuration stores."""
    W, V, S = cfg["width"], cfg["vocab"], cfg.get("streams")
    shapes = {"embed": (V, W), "head": (V, W), "final.norm": (W,), "final.norm.b": (W,)}
    for i, layer in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", layer["mixer"], layer.get("mlp")
        for n in ("1", "2") if f else ("1",):
            shapes.update({f"{p}norm{n}": (W,), f"{p}norm{n}.b": (W,)})
            if S:
                shapes.update({f"{p}hc{n}.in": (S,), f"{p}hc{n}.out": (S,), f"{p}hc{n}.mix": (S, S)})
        if layer["type"] == "attention":
            H, G, d = m["heads"], m.get("kv_heads", m["heads"]), m["dim"]
            shapes.update({p + "mix.q": (H * d, W), p + "mix.k": (G * d, W), p + "mix.g": (H, W), p + "mix.o": (W, H * d)})
        else:
            x, q = m["left"], p + "mix.left."
            H, G, d, dv = x["heads"], x.get("kv_heads", x["heads"]), x["dim"], x.get("vdim", x["dim"])
            for r, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
                shapes.update({q + r: (n, W), f"{q}{r}.b": (n,)})
            shapes.update({q + "q.norm": (d,), q + "k.norm": (d,), q + "rel": (x["bias_rows"], H), q + "g": (H * dv, W), q + "o": (W, H * dv)})
            x, q = m["right"], p + "mix.right."
            H, d, dv = x["heads"], x["dim"], x.get("vdim", x["dim"])
            shapes.update({q + "q": (H * d, W), q + "k": (H * d, W), q + "v": (H * dv, W), q + "g": (H * dv, W), q + "o": (W, H * dv)})
        if f:
            shapes.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"])})
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
        elif last == "mix" and ".hc" in name:
            z = 0.8 * torch.eye(shape[0]) + 0.25 * z       # not symmetric: [from, to] matters
        elif last in ("in", "out"):
            z = 1.0 / shape[0] + 0.5 * z if last == "in" else 1.0 + 0.4 * z
        elif last == "rel":
            z = 1.5 * z
        elif last == "b":
            z = 0.3 * z
        elif len(shape) == 1:
            z = 1.0 + 0.15 * z
            if name.endswith("left.q.norm"):
                z = z * sharpen
        else:
            z = z / math.sqrt(shape[-1]) * (1.5 if last == "up" else 1.0)
            if name.endswith(".mix.q"):
                z = z * sharpen
        out[name] = z.to(torch.bfloat16)
    return out


def random_prompts(cfg, lengths, seed):
    gen = torch.Generator().manual_seed(1000 + seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=gen).tolist() for n in lengths]


def random_config(seed):
    """A configuration drawn from odd sizes: widths off the multiples of 8, head counts that do not divide alike, tables of
    few and of many rows, with and without each optional mechanism, loops and streams of any number."""
    gen = torch.Generator().manual_seed(9000 + seed)
    pick = lambda *values: values[int(torch.randint(0, len(values), (1,), generator=gen))]
    rot = lambda dim, factor: pick(None, _rot(pick(300.0, 10000.0, 1e6), pick(*[r for r in (2, 6, 16, 20, 48) if r <= dim]), factor))
    layers = []
    for _ in range(pick(1, 2, 3)):
        kv = pick(1, 2, 3)
        heads = kv * pick(1, 2, 4)
        dim = pick(6, 16, 20, 48, 64)
        if pick(0, 1):
            mixer = _attention(heads, kv, dim, pick(0.1, 0.3), pick(None, 5.0, 30.0), rot(dim, pick(None, 2.0, 7.5)))
        else:
            rows = pick(2, 5, 16, 40)
            d2 = pick(6, 16, 33, 48)
            decay = [pick(0.0, 0.5, 0.97, 0.9995, 1.0) for _ in range(pick(1, 2, 3))]
            mixer = _parallel(_left(heads, kv, dim, pick(5, 16, 40, 64), pick(0.1, 0.3), rows, rows // 2 + pick(1, 30, 200),
                                    pick(None, (0.3, 1), (0.1, 33))),
                              _right(decay, d2, pick(5, 16, 40), rot(d2, None)), pick(1.0, 0.3), pick(1.0, 1.7))
        layers.append((mixer, pick(None, 10, 24, 52)))
    start = pick(*range(len(layers)))
    loop = pick(None, (start, pick(*range(start + 1, len(layers) + 1)), pick(1, 2, 3)))
    return _config(pick(50, 131), pick(36, 50, 64, 72), layers, pick(None, 1, 2, 3, 4, 7), loop, pick(1.0, 4.0), pick(1.0, 0.5),
                   pick(1.0, 0.25, 3.0), pick(None, 12.0), pick(1e-5, 1e-6))
