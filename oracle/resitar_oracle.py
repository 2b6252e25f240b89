"""Plain, slow restatement of the Resitar decoder, one function per mechanism, for the tests.

Resitar is a decoder-only model given as a list of layers around several residual streams.  The embedding output is rms(E[token]) * w_embed,
and every one of the n streams starts as it.  A sublayer (mixer, then feed-forward) with the numbers a [n], b [n] and M [n, n]:

    u = sum_s a_s x_s;   y = sublayer(rms(u) * w);   x_t <- sum_s M[s, t] x_s + b_t y     (all streams from the old ones)

At the end x = sum_s x_s and the logits are E . (rms(x) * w_final).  A run of layers may be looped: it runs `times` times in a row with the
same weights and a cache and state of its own per pass.

Both mixer types are two mixers side by side on the same input h, left_scale * left + right_scale * right.

* "parallel", left: grouped-query softmax attention; q and k are biased projections rotated on half-split pairs (i, i + dims/2), the VALUE
  of a token is its key before the rotation (there is no value projection); position i sees j <= i of the same chunk, floor(i / size) =
  floor(j / size); the heads times sigmoid(G h) elementwise, then the biased output projection.
  Right: a state-space recurrence with one decay per head.  in . h = z | x | B | C | dt; x, B and C pass a causal convolution (with bias) and
  silu; d = softplus(dt + dt_bias), alpha = exp(-exp(A_log) d); head a uses group a // (heads / groups):
      S <- alpha S + d B x^T;   y = S^T C + D x.
  y * silu(z), RMS-normed in norm_groups equal parts, times a gain, projected.
* "parallel_2", left: grouped-query causal softmax attention with biased q, k, v, rotated on interleaved pairs (2i, 2i+1) with
  wavelength-dependent interpolation of the frequencies (below), the same gate, an unbiased output projection.
  Right: time mixing.  With h' the previous token's h (zeros at the start), r, k, v, g, w each read their own blend h + (h' - h) * mu.  The
  decay is exp(-exp(W2 tanh(W1 blend_w) + w0)) per head and key channel; per head
      o = (S + diag(u) k v^T)^T r;   S <- diag(decay) S + k v^T.
  Each head's o divided by its root mean square, times a gain per channel, times silu(G blend_g), projected.

Interpolated frequencies (factor, original, fast, slow): f_i = base^(-2i/dims); with turn(t) = dims ln(original / (2 pi t)) / (2 ln base),
lo = max(floor(turn(fast)), 0) and hi = min(ceil(turn(slow)), dims - 1), a ramp from 0 at index lo to 1 at hi blends f_i with f_i / factor,
and cosines and sines are multiplied by 0.1 ln(factor) + 1.

Feed-forward: silu(gate) * up, dense or as experts: logits R h + b, the `top` largest, weighted by the softmax over the chosen logits.

Nothing here shares code with the engine.  Tensors go in as a dict of torch tensors under the checkpoint's names.  `Stepper` runs token by
token from explicit state; `forward` feeds a whole sequence through it.
"""
from __future__ import annotations

import math

import torch


def rms_norm(x: torch.Tensor, gain, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def silu(x: torch.Tensor) -> torch.Tensor:
    return x * torch.sigmoid(x)


def streams_in(xs: torch.Tensor, a: torch.Tensor) -> torch.Tensor:
    """xs [n, W]."""
    return (a[:, None] * xs).sum(0)


def streams_out(xs: torch.Tensor, mix: torch.Tensor, b: torch.Tensor, y: torch.Tensor) -> torch.Tensor:
    """mix [from, to]."""
    return mix.T @ xs + b[:, None] * y[None, :]


def frequencies(rot: dict):
    """-> (list of dims/2 angular frequencies, factor on cosines and sines)."""
    dims, base = rot["dims"], float(rot["base"])
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turn(t):
        return dims * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo, hi = max(math.floor(turn(sc["fast"])), 0), min(math.ceil(turn(sc["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / sc["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x: torch.Tensor, pos: int, rot: dict, halves: bool) -> torch.Tensor:
    """x [heads, dim]; the first rot["dims"] entries of every head turn, half-split or interleaved pairs."""
    f, mul = frequencies(rot)
    ang = torch.tensor([pos * fi for fi in f], dtype=torch.float64)
    c, s = (torch.cos(ang) * mul).to(x.dtype), (torch.sin(ang) * mul).to(x.dtype)
    half, y = len(f), x.clone()
    ia, ib = (slice(0, half), slice(half, 2 * half)) if halves else (slice(0, 2 * half, 2), slice(1, 2 * half, 2))
    y[:, ia], y[:, ib] = x[:, ia] * c - x[:, ib] * s, x[:, ib] * c + x[:, ia] * s
    return y


def attention_step(q: torch.Tensor, keys: torch.Tensor, values: torch.Tensor, first: int, scale: float) -> torch.Tensor:
    """One head: q [dim] over keys [n, dim] and values [n, vdim], positions first .. n-1 seen."""
    return torch.softmax((keys[first:] @ q) * scale, 0) @ values[first:]


def conv_step(hist: torch.Tensor, x: torch.Tensor, taps_w: torch.Tensor, bias: torch.Tensor):
    """hist [taps - 1, C] the inputs before x [C] (oldest first); taps_w [C, taps], last column for x.  -> (new hist, output [C])."""
    ext = torch.cat([hist, x[None]], 0)
    return ext[1:], (taps_w.T * ext).sum(0) + bias


def ssm_step(S: torch.Tensor, x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, d, a_log, D):
    """One head: S [state, vdim], d the step size.  -> (S', y [vdim])."""
    S = torch.exp(-torch.exp(a_log) * d) * S + d * B[:, None] * x[None, :]
    return S, S.T @ C + D * x


def time_mix_step(S: torch.Tensor, r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor, u: torch.Tensor):
    """One head: S [dim, dim].  -> (S', o [dim])."""
    kv = k[:, None] * v[None, :]
    return decay[:, None] * S + kv, (S + u[:, None] * kv).T @ r


def part_norm(y: torch.Tensor, parts: int, eps: float) -> torch.Tensor:
    """Each of `parts` equal pieces divided by its own root mean square."""
    return rms_norm(y.reshape(parts, -1), 1.0, eps).reshape(-1)


def gated_ff(x: torch.Tensor, w: dict, pre: str) -> torch.Tensor:
    return w[pre + "down"] @ (silu(w[pre + "gate"] @ x) * (w[pre + "up"] @ x))


def route(z: torch.Tensor, top: int):
    """Logits z [experts] -> (expert indices, weights), lowest index first on ties."""
    idx = sorted(range(z.numel()), key=lambda e: (-float(z[e]), e))[:top]
    return idx, torch.softmax(z[idx], 0)


def moe_ff(x: torch.Tensor, w: dict, pre: str, mlp: dict) -> torch.Tensor:
    idx, wt = route(w[pre + "router"] @ x + w[pre + "router.b"], mlp["router"]["top"])
    out = torch.zeros_like(x)
    for e, s in zip(idx, wt):
        out = out + s * gated_ff(x, w, "%se%d." % (pre, e))
    return out


def run_order(cfg: dict) -> list:
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return list(range(n))
    return list(range(lp["start"])) + list(range(lp["start"], lp["stop"])) * lp["times"] + list(range(lp["stop"], n))


class Stepper:
    """Token-by-token evaluation from explicit state, one per layer run."""

    def __init__(self, cfg: dict, w: dict, dtype=torch.float64):
        self.cfg, self.dtype = cfg, dtype
        self.w = {k: v.to(dtype) for k, v in w.items()}
        self.order = run_order(cfg)
        self.state = [dict() for _ in self.order]
        self.pos = 0
        self.trace = []          # sum of the streams after every layer run of the last token

    def attention(self, st, h, m, p, halves, eps):
        w, H, G, D = self.w, m["heads"], m["kv_heads"], m["dim"]
        q = (w[p + "q"] @ h + w[p + "q.b"]).reshape(H, D)
        k = (w[p + "k"] @ h + w[p + "k.b"]).reshape(G, D)
        v = k if halves else (w[p + "v"] @ h + w[p + "v.b"]).reshape(G, m["vdim"])
        if m.get("rot"):
            q, k = rotate(q, self.pos, m["rot"], halves), rotate(k, self.pos, m["rot"], halves)
        st["k"] = torch.cat([st["k"], k[None]]) if "k" in st else k[None]
        st["v"] = torch.cat([st["v"], v[None]]) if "v" in st else v[None]
        size = (m.get("mask") or {}).get("size", 0)
        first = self.pos // size * size if size else 0
        o = torch.cat([attention_step(q[a], st["k"][:, a // (H // G)], st["v"][:, a // (H // G)], first, m["scale"]) for a in range(H)])
        y = w[p + "o"] @ (o * torch.sigmoid(w[p + "g"] @ h))
        return y + w[p + "o.b"] if halves else y

    def ssm(self, st, h, m, p, eps):
        w, H, V, N, G = self.w, m["heads"], m["vdim"], m["state"], m["groups"]
        inner = H * V
        z, xbc, dt = torch.split(w[p + "in"] @ h, [inner, inner + 2 * G * N, H])
        cw = w[p + "conv"]
        hist = st.get("conv", torch.zeros(cw.shape[1] - 1, cw.shape[0], dtype=self.dtype))
        st["conv"], c = conv_step(hist, xbc, cw, w[p + "conv.b"])
        x, B, C = torch.split(silu(c), [inner, G * N, G * N])
        d = torch.nn.functional.softplus(dt + w[p + "dt_bias"], threshold=1e9)
        if "S" not in st:
            st["S"] = [torch.zeros(N, V, dtype=self.dtype) for _ in range(H)]
        outs = []
        for a in range(H):
            g = a // (H // G)
            st["S"][a], y = ssm_step(st["S"][a], x[a * V:(a + 1) * V], B[g * N:(g + 1) * N], C[g * N:(g + 1) * N], d[a], w[p + "A_log"][a], w[p + "D"][a])
            outs.append(y)
        return w[p + "o"] @ (part_norm(torch.cat(outs) * silu(z), m["norm_groups"], eps) * w[p + "norm"])

    def time_mix(self, st, h, m, p, eps):
        w, H, D = self.w, m["heads"], m["dim"]
        prev = st.get("h", torch.zeros_like(h))
        st["h"] = h
        b = {s: h + (prev - h) * w[p + "mu." + s] for s in "rkvgw"}
        r, k, v = ((w[p + s] @ b[s]).reshape(H, D) for s in "rkv")
        gate = silu(w[p + "g"] @ b["g"])
        decay = torch.exp(-torch.exp(w[p + "w2"] @ torch.tanh(w[p + "w1"] @ b["w"]) + w[p + "w0"])).reshape(H, D)
        if "S" not in st:
            st["S"] = [torch.zeros(D, D, dtype=self.dtype) for _ in range(H)]
        outs = []
        for a in range(H):
            st["S"][a], o = time_mix_step(st["S"][a], r[a], k[a], v[a], decay[a], w[p + "u"].reshape(H, D)[a])
            outs.append(rms_norm(o, 1.0, eps))
        return w[p + "o"] @ (torch.cat(outs) * w[p + "norm"] * gate)

    def mixer(self, st, L, h, pre, eps):
        m = L["mixer"]
        if L["type"] == "parallel":
            left, right = self.attention(st, h, m["left"], pre + "left.", True, eps), self.ssm(st, h, m["right"], pre + "right.", eps)
        elif L["type"] == "parallel_2":
            left, right = self.attention(st, h, m["left"], pre + "left.", False, eps), self.time_mix(st, h, m["right"], pre + "right.", eps)
        else:
            raise ValueError("mixer type %r" % L["type"])
        return m["left_scale"] * left + m["right_scale"] * right

    def step(self, token: int) -> torch.Tensor:
        """Appends one token; returns its logits."""
        cfg, w, eps = self.cfg, self.w, self.cfg["norm"]["eps"]
        x = rms_norm(w["embed"][token], w["embed.norm"], eps)
        xs = x[None].repeat(cfg["streams"], 1)
        self.trace = []
        for st, i in zip(self.state, self.order):
            L, p = cfg["layers"][i], "l%d." % i
            h = rms_norm(streams_in(xs, w[p + "hc1.in"]), w[p + "norm1"], eps)
            xs = streams_out(xs, w[p + "hc1.mix"], w[p + "hc1.out"], self.mixer(st, L, h, p + "mix.", eps))
            mlp = L.get("mlp")
            if mlp:
                h = rms_norm(streams_in(xs, w[p + "hc2.in"]), w[p + "norm2"], eps)
                y = gated_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, w, p + "mlp.", mlp)
                xs = streams_out(xs, w[p + "hc2.mix"], w[p + "hc2.out"], y)
            self.trace.append(xs.sum(0))
        self.pos += 1
        return w["embed"] @ rms_norm(xs.sum(0), w["final.norm"], eps)

    def greedy(self, prompt, n: int):
        """Feeds the prompt, then n times the most likely token (lowest index on ties); returns the n tokens."""
        for t in prompt:
            y = self.step(int(t))
        out = []
        for _ in range(n):
            out.append(int(torch.argmax(y)))
            y = self.step(out[-1])
        return out


def forward(cfg: dict, w: dict, tokens, dtype=torch.float64):
    """-> (logits [T, vocab], sum of the streams after every layer run [runs, T, W])."""
    s = Stepper(cfg, w, dtype)
    logits, traces = [], []
    for t in tokens:
        logits.append(s.step(int(t)))
        traces.append(torch.stack(s.trace))
    return torch.stack(logits), torch.stack(traces, 1)


def tensor_shapes(cfg: dict, rank: int = 8) -> dict:
    """name -> shape of every tensor a checkpoint of this config holds; rank = width of the decay's low-rank stage (only the tensors have it)."""
    W, V, n = cfg["width"], cfg["vocab"], cfg["streams"]
    sh = {"embed": (V, W), "embed.norm": (W,)}
    for i, L in enumerate(cfg["layers"]):
        p, a, b = "l%d." % i, L["mixer"]["left"], L["mixer"]["right"]
        l, r = p + "mix.left.", p + "mix.right."
        H, G, D = a["heads"], a["kv_heads"], a["dim"]
        HV = H * a["vdim"]
        sh[p + "norm1"] = (W,)
        sh.update({l + "q": (H * D, W), l + "q.b": (H * D,), l + "k": (G * D, W), l + "k.b": (G * D,), l + "g": (HV, W), l + "o": (W, HV)})
        if L["type"] == "parallel":
            sh[l + "o.b"] = (W,)
            inner, gn = b["heads"] * b["vdim"], b["groups"] * b["state"]
            C = inner + 2 * gn
            sh.update({r + "in": (inner + C + b["heads"], W), r + "conv": (C, b["conv"]), r + "conv.b": (C,), r + "dt_bias": (b["heads"],),
                       r + "A_log": (b["heads"],), r + "D": (b["heads"],), r + "norm": (inner,), r + "o": (W, inner)})
        else:
            sh.update({l + "v": (G * a["vdim"], W), l + "v.b": (G * a["vdim"],)})
            HD = b["heads"] * b["dim"]
            for s in "rkvgw":
                sh[r + "mu." + s] = (W,)
            for s in "rkvg":
                sh[r + s] = (HD, W)
            sh.update({r + "w1": (rank, W), r + "w2": (HD, rank), r + "w0": (HD,), r + "u": (b["heads"], b["dim"]), r + "norm": (HD,), r + "o": (W, HD)})
        mlp, f = L.get("mlp"), p + "mlp."
        if mlp:
            sh[p + "norm2"] = (W,)
            if mlp["kind"] == "dense":
                sh.update({f + "gate": (mlp["ff"], W), f + "up": (mlp["ff"], W), f + "down": (W, mlp["ff"])})
            else:
                F, E = mlp["expert"]["ff"], mlp["router"]["experts"]
                for e in range(E):
                    sh.update({"%se%d.gate" % (f, e): (F, W), "%se%d.up" % (f, e): (F, W), "%se%d.down" % (f, e): (W, F)})
                sh.update({f + "router": (E, W), f + "router.b": (E,)})
        for q in (1, 2) if mlp else (1,):
            sh.update({p + "hc%d.in" % q: (n,), p + "hc%d.out" % q: (n,), p + "hc%d.mix" % q: (n, n)})
    sh["final.norm"] = (W,)
    return sh


def random_weights(cfg: dict, seed: int, rank: int = 8, router_spread: float = 2.0) -> dict:
    """bf16-representable random weights; the router's rows are spread so that choices are rarely close."""
    gen = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg, rank).items():
        last = name.rsplit(".", 1)[-1]
        randn = torch.randn(shape, generator=gen)
        if "norm" in name:
            t = 1.0 + 0.2 * randn
        elif ".hc" in name:
            n = cfg["streams"]
            t = {"in": 1.0 / n + 0.3 * randn, "out": 1.0 + 0.3 * randn, "mix": (0.8 * torch.eye(n) if last == "mix" else 0) + 0.25 * randn}[last]
        elif ".mu." in name:
            t = torch.rand(shape, generator=gen)
        elif last == "A_log":
            t = torch.log(0.3 + 2.0 * torch.rand(shape, generator=gen))
        elif last == "dt_bias":
            t = randn - 2.0
        elif last == "w0":
            t = randn - 2.5
        elif last in ("D", "u"):
            t = randn
        elif last == "b":
            t = 0.3 * randn
        elif last == "conv":
            t = 0.5 * randn
        elif last == "router":
            t = router_spread * randn / math.sqrt(shape[-1])
        elif name == "embed":
            t = randn / math.sqrt(shape[-1])
        else:
            t = randn / math.sqrt(shape[-1])
        w[name] = t.to(torch.bfloat16).to(torch.float32)
    return w
