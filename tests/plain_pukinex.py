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
    """[heads, P, J] of rel[bucket(p - j), head] (0 where j > p, which nobody sees)."""
    rows = [[bucket(max(int(p) - int(j), 0), rel.shape[0], reach) for j in keys] for p in queries]
    return rel[torch.tensor(rows)].permute(2, 0, 1)


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
