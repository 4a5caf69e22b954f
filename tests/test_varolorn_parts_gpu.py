"""The mechanisms the Varolorn design brought, each alone against its plain function: residual streams (read, norm, write, the
block around them), the norm stored around zero, pair rows in the embedding and their state, the relu-gated feed-forward in
every contraction form, the short convolution with bias and silu, the norm in parts behind a gate, the Mamba-2 recurrence (an
input made so that the FIRST token decides an output hundreds of steps later), and attention with biases, normed heads,
distance buckets, stretches, a gate per head and mixed values (every kernel that takes it, heads padded or not; inputs made so
that ONE marked key, or one bucket of the table, decides the last query: just inside and just outside its stretch, at page
borders, in a prompt step and as a single token)."""
import numpy as np
import pytest
import torch

import plain_varolorn as P
from test_parts_gpu import close, load, rnd, run_mixer

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def k():
    from zinfer_b200 import kernels
    kernels.require_cuda()
    return kernels


def f64(t):
    return t.numpy().astype(np.float64)


class Ctx:
    """The little of a step context that a norm or a feed-forward reads."""

    def __init__(self, k, dtype, n, decode=False):
        self.dtype, self.device, self.status = dtype, torch.device("cuda"), k.status_word(torch.device("cuda"))
        self.n_tokens, self.is_decode, self._memo, self.shared = n, decode, {}, {}

    def memo(self, key, make):
        if key not in self._memo:
            self._memo[key] = make()
        return self._memo[key]


# ------------------------------------------------------------------------------- norms and streams

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("dim", [38, 192, 2048])
def test_norm_with_a_weight_around_zero(k, dtype, dim):
    from zinfer_b200.parts import RMSNorm
    t = {"w": rnd((dim,), 1, dtype, 0.5)}
    norm = load(RMSNorm(dim, 1e-3, "w", one_plus=True), t, dtype)
    x = rnd((9, dim), 2, torch.float32, 0.1)                  # small rows: where the eps sits shows
    ref = P.plus_one_norm(f64(x), f64(t["w"]), 1e-3)
    close(norm.forward(Ctx(k, dtype, 9), x.cuda()), ref, dtype, "all rows")
    close(norm.pending(Ctx(k, dtype, 9), x.cuda()).tensor(), ref, dtype, "pending")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,dim", [(1, 64), (2, 38), (3, 200), (4, 2048), (5, 128), (6, 33), (2, 5000), (3, 9000), (2, 1000)])
def test_streams_are_read_and_written(k, dtype, S, dim):
    """Reading (all rows, chosen rows, the plain sum), writing without a norm behind it, and writing with one."""
    n, eps = 7, 1e-3
    X, y = rnd((S, n, dim), 1, torch.float32, 0.3), rnd((n, dim), 2, torch.float32)
    a, w = rnd((S,), 3, torch.float32), 1.0 + rnd((dim,), 4, torch.float32, 0.3)
    mix, out = rnd((S, S), 5, torch.float32), rnd((S,), 6, torch.float32)
    ref = P.rms(P.stream_read(f64(X), f64(a)), eps) * f64(w)
    close(k.stream_norm(X.cuda(), a.cuda(), w.cuda(), eps, dtype), ref, dtype, "read")
    rows = torch.tensor([5, 0, 2], dtype=torch.int32, device="cuda")
    close(k.stream_norm(X.cuda(), None, w.cuda(), eps, dtype, rows), (P.rms(f64(X).sum(0), eps) * f64(w))[[5, 0, 2]], dtype, "sum, chosen rows")
    new = P.stream_write(f64(X), f64(mix), f64(out), f64(y))
    x = X.clone().cuda()
    assert k.stream_step(x, y.cuda(), mix.cuda(), out.cuda()) is None
    close(x, new, torch.float32, "write")
    for read in (a, None):
        x = X.clone().cuda()
        h = k.stream_step(x, y.cuda(), mix.cuda(), out.cuda(), None if read is None else read.cuda(), w.cuda(), eps, dtype)
        close(x, new, torch.float32, "write with a norm behind it")
        u = P.stream_read(new, f64(read) if read is not None else np.ones(S))
        close(h, P.rms(u, eps) * f64(w), dtype, "the next sublayer's rows")
        again = k.stream_norm(x, None if read is None else read.cuda(), w.cuda(), eps, dtype)
        close(again, P.rms(u, eps) * f64(w), dtype, "the same rows read afterwards")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("S,with_ffn", [(1, True), (3, True), (4, False)])
def test_stream_block(k, dtype, S, with_ffn):
    """Two blocks in a row, the second's norm made by the first's last pass or by itself: both must agree with the plain
    functions.  The mixer is a plain contraction."""
    from zinfer_b200.parts import Mixer, ReluGLU, StreamBlock, StreamNorm, WeightSpec, linear

    D, F, n, eps = 64, 48, 11, 1e-5

    class Map(Mixer):
        def __init__(self, name):
            self.name = name

        def weight_specs(self):
            return [WeightSpec(self.name, (D, D))]

        def load(self, weights, dt, device):
            self.w = weights[self.name]

        def forward(self, ctx, call, xn, out, accumulate):
            linear(xn, self.w, out=out, accumulate=accumulate)

    t, blocks = {}, []
    for i in range(2):
        for q in (1, 2):
            t |= {f"{i}norm{q}": rnd((D,), 10 * i + q, dtype, 0.3), f"{i}in{q}": rnd((S,), 20 + 10 * i + q, dtype),
                  f"{i}mix{q}": rnd((S, S), 40 + 10 * i + q, dtype), f"{i}out{q}": rnd((S,), 60 + 10 * i + q, dtype)}
        t |= {f"{i}m": rnd((D, D), 80 + i, dtype, D ** -0.5), f"{i}g": rnd((F, D), 82 + i, dtype, D ** -0.5),
              f"{i}u": rnd((F, D), 84 + i, dtype, D ** -0.5), f"{i}d": rnd((D, F), 86 + i, dtype, F ** -0.5)}
        norm = [StreamNorm(D, eps, f"{i}norm{q}", S, read_name=f"{i}in{q}", one_plus=True) for q in (1, 2)]
        ffn = (norm[1], ReluGLU(D, F, f"{i}g", f"{i}u", f"{i}d"), (f"{i}mix2", f"{i}out2")) if with_ffn else ()
        blocks.append(load(StreamBlock(norm[0], Map(f"{i}m"), (f"{i}mix1", f"{i}out1"), *ffn), t, dtype))
    X = rnd((S, n, D), 90, torch.float32)
    w = {name: f64(v) for name, v in t.items()}
    ref = f64(X)
    for i in range(2):
        h = P.plus_one_norm(P.stream_read(ref, w[f"{i}in1"]), w[f"{i}norm1"], eps)
        ref = P.stream_write(ref, w[f"{i}mix1"], w[f"{i}out1"], h @ w[f"{i}m"].T)
        if with_ffn:
            h = P.plus_one_norm(P.stream_read(ref, w[f"{i}in2"]), w[f"{i}norm2"], eps)
            ref = P.stream_write(ref, w[f"{i}mix2"], w[f"{i}out2"], P.gated_relu(h, w[f"{i}g"], w[f"{i}u"], w[f"{i}d"]))
    for chained in (True, False):
        x, ctx = X.clone().cuda(), Ctx(k, dtype, n)
        made = blocks[0].forward_chained(ctx, None, x, None, blocks[1].entry_norm() if chained else None)
        assert (made is not None) == chained
        blocks[1].forward_chained(ctx, None, x, made, None)
        close(x, ref, dtype, f"two blocks, chained {chained}")
    with pytest.raises(ValueError):
        StreamBlock(norm[0], Map("m"), ("a", "b"), norm[1])


# ------------------------------------------------------------------------------- pair rows

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("buckets,mul_prev,mul_cur,copies", [(37, 5, 11, None), (1, 3, 7, 1), (1000, 2147483659, 40503, 3), (5, -3, 2, 1)])
def test_pair_rows_in_steps(k, dtype, buckets, mul_prev, mul_cur, copies):
    """Two sequences in portions (down to one token) whose slots are then used again: the token before comes from the step
    or from the state, the first token takes the last row."""
    from zinfer_b200.engine.context import StepContext, pack_batch
    from zinfer_b200.parts import TokenEmbedding
    V, D = 60, 40
    t = {"e": rnd((V, D), 1, dtype), "b": rnd((buckets + 1, D), 2, dtype)}
    emb = load(TokenEmbedding(V, D, "e", scale=1.5, bigram=("b", buckets, mul_prev, mul_cur), copies=copies), t, dtype)
    state = torch.full((5, 1), 41, dtype=torch.int32, device="cuda")          # whatever a former user left
    status = k.status_word(torch.device("cuda"))
    for seed, slots in ((3, [3, 1]), (4, [1, 3])):
        toks = [np.random.default_rng(seed + b).integers(0, V, n).tolist() for b, n in enumerate((17, 12))]
        got = [[], []]
        at = [0, 0]
        for sizes in ((4, 1), (2, 3), (1, 1), (1, 1), (8, 2), (1, 4)):
            part = [toks[b][at[b]:at[b] + sizes[b]] for b in range(2)]
            buf = torch.from_numpy(pack_batch(slots, at, part)).cuda()
            ctx = StepContext(dtype, torch.device("cuda"), status, buf, sum(sizes), 2, list(sizes), 32, starts=at)
            x = emb.forward(ctx, ctx.tokens, state=state)
            assert x.shape == ((sum(sizes), D) if copies is None else (copies, sum(sizes), D))
            for c in range(copies or 0):
                assert torch.equal(x[c], x[0])
            x = x if copies is None else x[0]
            got[0].append(x[:sizes[0]].cpu())
            got[1].append(x[sizes[0]:].cpu())
            at = [at[b] + sizes[b] for b in range(2)]
        for b in range(2):
            ref = P.embed_rows(toks[b][:at[b]], f64(t["e"]), 1.5, (f64(t["b"]), buckets, mul_prev, mul_cur))
            close(torch.cat(got[b]), ref, torch.float32, f"sequence {b}")
    assert int(status.item()) == 0 and state[[0, 2, 4]].eq(41).all()


# ------------------------------------------------------------------------------- feed-forward

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [1, 5, 16, 17, 40, 64, 65, 129, 300])
@pytest.mark.parametrize("D,F", [(64, 128), (256, 512), (38, 22), (64, 24)])
def test_relu_gated_feed_forward(k, dtype, rows, D, F):
    from zinfer_b200.parts import ReluGLU, RMSNorm
    t = {"g": rnd((F, D), 1, dtype, D ** -0.5), "u": rnd((F, D), 2, dtype, D ** -0.5), "d": rnd((D, F), 3, dtype, F ** -0.5),
         "n": 1.0 + rnd((D,), 4, dtype, 0.2)}
    ffn, norm = load(ReluGLU(D, F, "g", "u", "d"), t, dtype), load(RMSNorm(D, 1e-5, "n"), t, dtype)
    x, ctx = rnd((rows, D), 5, dtype), Ctx(k, dtype, rows)
    out = torch.empty((rows, D), device="cuda")
    ffn.forward(ctx, x.to(dtype).cuda(), out, False)
    close(out, P.gated_relu(f64(x), *(f64(t[n]) for n in "gud")), dtype, "tensor")
    base = out.clone()
    ffn.forward(ctx, norm.pending(ctx, x.cuda()), out, True)
    close(out - base, P.gated_relu(P.rms(f64(x), 1e-5) * f64(t["n"]), *(f64(t[n]) for n in "gud")), dtype, "pending norm, summed")


# ------------------------------------------------------------------------------- the recurrence

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("inner,parts,skip", [(48, 1, 9), (48, 4, 16), (40, 8, 3), (1024, 2, 0), (4096, 1, 8), (9000, 1, 4), (33, 3, 1)])
def test_gate_then_norm_in_parts(k, dtype, inner, parts, skip):
    y, z = rnd((7, inner), 1, torch.float32, 0.2), rnd((7, inner + skip), 2, torch.float32, 2.0)
    w = 1.0 + rnd((inner,), 3, torch.float32, 0.3)
    ref = P.gated_group_norm(f64(y), f64(z)[:, :inner], f64(w), parts, 1e-3)
    close(k.gated_group_norm(y.cuda(), z.cuda()[:, :inner], w.cuda(), parts, 1e-3, dtype), ref, dtype, "gate and norm")


def ssm_tensors(D, H, e, N, G, K, dtype, seed):
    ch = H * e + 2 * G * N
    return {"in": rnd((H * e + ch + H, D), seed, dtype, D ** -0.5), "conv": rnd((ch, K), seed + 1, dtype, K ** -0.5),
            "conv.b": rnd((ch,), seed + 2, dtype, 0.3), "dt_bias": rnd((H,), seed + 3, dtype) - 1.0, "A_log": rnd((H,), seed + 4, dtype) - 1.0,
            "D": 1.0 + rnd((H,), seed + 5, dtype, 0.3), "norm": 1.0 + rnd((H * e,), seed + 6, dtype, 0.3),
            "o": rnd((D, H * e), seed + 7, dtype, (H * e) ** -0.5)}


def make_ssm(D, H, e, N, G, K, parts, t, dtype, eps=1e-5):
    from zinfer_b200.parts import Mamba2
    t = dict(t)
    for n in ("dt_bias", "A_log"):
        t[n] = t[n].to(dtype).float()
    return load(Mamba2(D, H, e, N, G, K, parts, "in", "conv", "conv.b", "dt_bias", "A_log", "D", "norm", "o", norm_eps=eps), t, dtype)


def plain_ssm(x, t, dtype, H, e, N, G, K, parts, eps=1e-5):
    w = {n: f64(a) for n, a in t.items()}
    for n in ("dt_bias", "A_log"):
        w[n] = f64(t[n].to(dtype).float())
    return P.mamba2(f64(x), w, {"heads": H, "vdim": e, "state": N, "groups": G, "norm_groups": parts}, eps)


SSM_SHAPES = [(48, 3, 10, 8, 1, 3, 2), (64, 4, 16, 16, 4, 4, 4), (32, 1, 6, 4, 1, 1, 1), (38, 5, 3, 7, 5, 3, 5), (128, 4, 32, 64, 2, 4, 4),
              (64, 2, 64, 128, 1, 2, 1), (64, 2, 40, 200, 2, 5, 2), (256, 8, 64, 128, 2, 4, 2)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,H,e,N,G,K,parts", SSM_SHAPES)
@pytest.mark.parametrize("prompts", [(70, 17, 1), (2, 3, 12)])
def test_recurrence_alone(k, dtype, D, H, e, N, G, K, parts, prompts):
    """Three unequal sequences in one batch: a prompt step, then single tokens: the convolution's inputs and the state pass
    from one to the other, whatever of the taps the prompt filled."""
    t = ssm_tensors(D, H, e, N, G, K, dtype, 10)
    mixer = make_ssm(D, H, e, N, G, K, parts, t, dtype)
    xs = [rnd((n, D), 20 + b, dtype) for b, n in enumerate((90, 37, 12))]
    outs = run_mixer(k, mixer, dtype, xs, list(prompts))
    for b, x in enumerate(xs):
        close(outs[b], plain_ssm(x, t, dtype, H, e, N, G, K, parts), dtype, f"sequence {b}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [300, 100, 2, 1])
def test_recurrence_keeps_the_first_token_for_hundreds_of_steps(k, dtype, prompt):
    """Slow decays and keys that all tokens but the first two have tiny: every later output is what the first tokens left in
    the state."""
    D, H, e, N, G, K, parts = 32, 2, 8, 8, 1, 3, 1
    t = ssm_tensors(D, H, e, N, G, K, dtype, 30)
    inner = H * e
    t["in"][2 * inner:2 * inner + N, D // 2:] = 0.0            # keys read the first half of the input only
    t["conv.b"][inner:inner + N] = 0.0
    t["A_log"][:] = -5.0
    t["D"][:] = 0.0
    mixer = make_ssm(D, H, e, N, G, K, parts, t, dtype)
    x = rnd((300, D), 31, dtype)
    x[1:, :D // 2] *= 2.0 ** -10
    ref = plain_ssm(x, t, dtype, H, e, N, G, K, parts)
    without = x.clone()
    without[0, :D // 2] = -x[0, :D // 2].flip(0)
    assert np.abs(ref[-1] - plain_ssm(without, t, dtype, H, e, N, G, K, parts)[-1]).max() > 0.1 * np.abs(ref).max()
    outs = run_mixer(k, mixer, dtype, [x], [prompt], page=16)
    close(outs[0], ref, dtype, f"prompt of {prompt}")


def test_a_batch_changes_no_bit_of_the_recurrence(k):
    """A sequence alone and beside others: the same bits."""
    D, H, e, N, G, K, parts = 64, 4, 16, 16, 2, 4, 2
    t = ssm_tensors(D, H, e, N, G, K, torch.float32, 50)
    mixer = make_ssm(D, H, e, N, G, K, parts, t, torch.float32)
    xs = [rnd((n, D), 60 + b, torch.float32) for b, n in enumerate((40, 33, 50))]
    together = run_mixer(k, mixer, torch.float32, xs, [30, 20, 45])
    alone = run_mixer(k, mixer, torch.float32, [xs[1]], [20])
    assert torch.equal(together[1], alone[0])


# ------------------------------------------------------------------------------- attention

def att_tensors(D, H, G, d, e, rows, dtype, seed):
    return {"q": rnd((H * d, D), seed, dtype, D ** -0.5), "k": rnd((G * d, D), seed + 1, dtype, D ** -0.5),
            "v": rnd((G * e, D), seed + 2, dtype, D ** -0.5), "o": rnd((D, H * e), seed + 3, dtype, (H * e) ** -0.5),
            "q.b": rnd((H * d,), seed + 4, dtype, 0.3), "k.b": rnd((G * d,), seed + 5, dtype, 0.3), "v.b": rnd((G * e,), seed + 6, dtype, 0.3),
            "o.b": rnd((D,), seed + 7, dtype, 0.3), "q.norm": 1.0 + rnd((d,), seed + 8, dtype, 0.2), "k.norm": 1.0 + rnd((d,), seed + 9, dtype, 0.2),
            "rel": rnd((rows, H), seed + 10, dtype), "g": rnd((H, D), seed + 11, dtype, 2.0 * D ** -0.5),
            "vmix": rnd((), seed + 12, dtype, 0.1) + 0.5}


def make_att(D, H, G, d, e, scale, bias_max, size, t, dtype, eps=1e-5, pad=True, v_mix=None, split_keys=0):
    from zinfer_b200.parts import GqaAttention
    t = {n: (a.to(dtype).float() if n in ("vmix", "q.norm", "k.norm") else a) for n, a in t.items()}
    return load(GqaAttention(D, H, G, d, "q", "k", "v", "o", "q.norm", "k.norm", norm_eps=eps, scale=scale, value_dim=e, pad_heads=pad,
                             bias_names=("q.b", "k.b", "v.b", "o.b"), distance_rows=("rel", bias_max), chunk=size, head_gate_name="g",
                             value_mix=None if v_mix is None else ("vmix", v_mix), split_keys=split_keys), t, dtype)


def plain_att(x, t, dtype, H, G, d, e, scale, bias_max, size, eps=1e-5, v_first=None):
    w = {n: f64(a.to(dtype).float() if n in ("vmix", "q.norm", "k.norm") else a) for n, a in t.items()}
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "scale": scale, "bias_max": bias_max, "mask": {"size": size} if size else None}
    return P.attention(f64(x), w, m, eps, v_first)


ATT_SHAPES = [  # D, H, G, d, e, scale, rows, bias_max, size, page
    (48, 4, 2, 16, 12, 0.3, 6, 9.5, 7, 16), (64, 8, 8, 8, 16, 0.35, 16, 24, 0, 16), (38, 5, 1, 10, 7, 0.4, 2, 13, 5, 16),
    (128, 8, 2, 64, 64, 0.12, 32, 50, 80, 64), (128, 6, 2, 64, 64, 0.15, 12, 200, 128, 64), (128, 4, 4, 64, 64, 0.12, 7, 33, 0, 64),
    (96, 4, 2, 24, 40, 0.2, 10, 60, 100, 64), (96, 6, 2, 72, 40, 0.12, 20, 90, 70, 64), (96, 2, 2, 128, 128, 0.1, 3, 40, 64, 64),
    (128, 8, 1, 64, 64, 0.12, 8, 30, 1, 64), (64, 20, 1, 64, 64, 0.12, 8, 70, 50, 64), (64, 16, 2, 64, 32, 0.14, 16, 300, 150, 64),
    (64, 2, 1, 64, 160, 0.12, 16, 30, 90, 64), (512, 16, 4, 64, 64, 0.12, 24, 100, 200, 64)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,H,G,d,e,scale,rows,bias_max,size,page", ATT_SHAPES)
@pytest.mark.parametrize("prompts", [(270, 17, 1), (65, 128, 2)])
def test_attention_alone(k, dtype, D, H, G, d, e, scale, rows, bias_max, size, page, prompts):
    """Three unequal sequences: a prompt step, then single tokens, over many stretches and pages (and a stretch's end inside
    a prompt, at its last token, between two single tokens).  The shapes reach every kernel: general, mma.sync and tcgen05
    prompt, single-token with one cut and several, heads padded to 64 and 128."""
    t = att_tensors(D, H, G, d, e, rows, dtype, 40)
    mixer = make_att(D, H, G, d, e, scale, bias_max, size, t, dtype)
    padded = dtype == torch.bfloat16 and not (d == e and d in (64, 128)) and max(d, e) <= 128
    assert (mixer.run_head_dim, mixer.run_value_dim) == ((64, 64) if padded and max(d, e) <= 64 else (128, 128) if padded else (d, e))
    xs = [rnd((n, D), 50 + b, dtype, 1.5) for b, n in enumerate((300, 140, 9))]
    outs = run_mixer(k, mixer, dtype, xs, list(prompts), page=page)
    for b, x in enumerate(xs):
        close(outs[b], plain_att(x, t, dtype, H, G, d, e, scale, bias_max, size)[0], dtype, f"sequence {b}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,page", [(4, 2, 16, 16), (8, 2, 64, 64), (2, 2, 128, 64), (2, 1, 40, 64)])
@pytest.mark.parametrize("size,T,marks", [(100, 230, (199, 200, 201, 207, 208, 228)), (64, 192, (127, 128, 143, 144, 190)), (80, 161, (159, 0, 80)),
                                          (0, 260, (0, 15, 16, 63, 64, 191, 192, 258)), (300, 290, (0, 63, 64, 128, 288)), (70, 141, (139, 69, 70))])
def test_one_marked_key_decides_the_last_query(k, dtype, H, G, d, page, size, T, marks):
    """The last token's query matches the key of token `mark` alone.  Inside the last token's stretch that key decides the
    output; just outside (the last position of the stretch before, or the token a stretch earlier) it must not be seen at
    all.  The last token comes in a prompt step, alone behind a prompt, and behind many single tokens."""
    D = 2 * d
    t = att_tensors(D, H, G, d, d, 8, dtype, 70)
    t["k"][:, D // 2:] = 0.0
    t["v"][:, :D // 2] = 0.0
    t["q"] = t["k"].reshape(G, 1, d, D).expand(G, H // G, d, D).reshape(H * d, D).clone()
    for n in ("q.b", "k.b", "rel"):
        t[n] *= 0.0
    t["k.norm"] = t["q.norm"] = torch.ones(d)
    scale = (16.0 if d <= 40 else 40.0) / d
    mixer = make_att(D, H, G, d, d, scale, 20, size, t, dtype)
    for mark in marks:
        x = rnd((T, D), 71 + mark, dtype)
        x[T - 1, :D // 2] = x[mark, :D // 2]
        ref = plain_att(x, t, dtype, H, G, d, d, scale, 20, size)[0]
        other = x.clone()
        other[mark, D // 2:] = rnd((D // 2,), 72, dtype, 3.0)
        moved = plain_att(other, t, dtype, H, G, d, d, scale, 20, size)[0]
        seen = size == 0 or mark // size == (T - 1) // size
        alone = size > 0 and (T - 1) % size == 0
        assert seen == (np.abs(ref[-1] - moved[-1]).max() > 0.05 * np.abs(ref).max()) or alone, "the marked key does not decide the last query"
        for prompt in (T, T - 1, T - 30):
            outs = run_mixer(k, mixer, dtype, [x], [prompt], page=page)
            close(outs[0], ref, dtype, f"mark {mark}, prompt of {prompt}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,page", [(4, 2, 16, 16), (8, 2, 64, 64), (2, 2, 128, 64)])
@pytest.mark.parametrize("rows,bias_max,size", [(16, 100, 0), (7, 40, 150), (8, 16, 60), (4, 1000, 0)])
def test_one_bucket_of_the_table_decides(k, dtype, H, G, d, page, rows, bias_max, size):
    """Every bucket in turn gets a number that lifts its keys above all others: a bucket's edge that is off by one, a table
    that is scaled, or a head's column that is another's, moves the output by far more than rounding."""
    D, T = 64, 210
    t = att_tensors(D, H, G, d, d, rows, dtype, 90)
    for hot in range(rows):
        t["rel"] = torch.zeros((rows, H))
        for h in range(H):
            t["rel"][(hot + h) % rows, h] = 12.0
        mixer = make_att(D, H, G, d, d, d ** -0.5, bias_max, size, t, dtype)
        x = rnd((T, D), 91 + hot, dtype)
        ref = plain_att(x, t, dtype, H, G, d, d, d ** -0.5, bias_max, size)[0]
        outs = run_mixer(k, mixer, dtype, [x], [T - 25], page=page)
        close(outs[0], ref, dtype, f"bucket {hot}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,T", [(500, 760), (0, 700), (130, 300)])
@pytest.mark.parametrize("H,G,d,e,page", [(8, 2, 64, 64, 64), (4, 2, 16, 24, 16), (16, 1, 128, 128, 64)])
def test_single_tokens_with_the_keys_cut_between_blocks(k, dtype, H, G, d, e, page, size, T):
    """Cuts of 64 keys, counted from the stretch's start; the gate is then the merge kernel's."""
    D = 64
    t = att_tensors(D, H, G, d, e, 16, dtype, 110)
    mixer = make_att(D, H, G, d, e, 1.5 * d ** -0.5, 90, size, t, dtype, split_keys=64, pad=False)
    xs = [rnd((n, D), 120 + b, dtype) for b, n in enumerate((T, 70))]
    outs = run_mixer(k, mixer, dtype, xs, [T - 12, 3], page=page)
    for b, x in enumerate(xs):
        close(outs[b], plain_att(x, t, dtype, H, G, d, e, 1.5 * d ** -0.5, 90, size)[0], dtype, f"sequence {b}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,e,page", [(4, 2, 16, 12, 16), (8, 2, 64, 64, 64), (4, 2, 24, 40, 64), (6, 2, 72, 40, 64)])
@pytest.mark.parametrize("T,prompts", [(330, (300, 20)), (60, (40, 1))])
def test_values_mixed_with_a_first_layers(k, dtype, H, G, d, e, page, T, prompts):
    """The mixed values are what later tokens attend to, so the first layer's values of a token matter at its own step only."""
    D, size = 64, 45
    t = att_tensors(D, H, G, d, e, 8, dtype, 130)
    inner = make_att(D, H, G, d, e, d ** -0.5, 30, size, t, dtype, v_mix=False)
    first = [rnd((T, G, e), 131 + b, dtype, 2.0) for b in range(2)]
    table = torch.stack(first).to(dtype).cuda()

    from zinfer_b200.parts import Mixer

    class WithFirstValues(Mixer):
        capture_safe = True
        seqs = None

        def kv_request(self):
            return inner.kv_request()

        def forward(self, ctx, call, xn, out, accumulate):
            slots = ctx.seq_slot.long()[ctx.tok_seq.long()]       # run_mixer hands slots out in reverse: 2 - slot = sequence
            ctx.shared["first values"] = table[2 - slots, ctx.tok_pos.long()]
            inner.forward(ctx, call, xn, out, accumulate)

    xs = [rnd((T, D), 140 + b, dtype) for b in range(2)]
    outs = run_mixer(k, WithFirstValues(), dtype, xs, list(prompts), page=page)
    for b, x in enumerate(xs):
        ref = plain_att(x, t, dtype, H, G, d, e, d ** -0.5, 30, size, v_first=f64(first[b]))[0]
        close(outs[b], ref, dtype, f"sequence {b}")
    unmixed = plain_att(xs[0], t, dtype, H, G, d, e, d ** -0.5, 30, size)[0]
    assert np.abs(unmixed - plain_att(xs[0], t, dtype, H, G, d, e, d ** -0.5, 30, size, v_first=f64(first[0]))[0]).max() > 0.1


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_layer_leaves_its_unmixed_values(k, dtype):
    D, H, G, d, e = 64, 4, 2, 24, 40
    t = att_tensors(D, H, G, d, e, 8, dtype, 150)
    mixer = make_att(D, H, G, d, e, 0.2, 30, 20, t, dtype, v_mix=True)
    seen = []
    forward = mixer.forward

    def spy(ctx, *a):
        forward(ctx, *a)
        seen.append(ctx.shared["first values"].float().cpu().numpy())

    mixer.forward = spy
    x = rnd((50, D), 151, dtype)
    outs = run_mixer(k, mixer, dtype, [x], [45], page=64)
    ref, own = plain_att(x, t, dtype, H, G, d, e, 0.2, 30, 20)
    close(outs[0], ref, dtype, "output")
    close(torch.from_numpy(np.concatenate(seen)), own, dtype, "values left behind")


def test_what_does_not_go_together_is_refused():
    from zinfer_b200.parts import GqaAttention
    args = (64, 4, 2, 16, "q", "k", "v", "o")
    for bad in (dict(chunk=8, window=8), dict(chunk=-1), dict(chunk=8, talk_name="t"), dict(head_gate_name="g", own_kv=False),
                dict(distance_rows=("r", 9), qk_norm_span="all")):
        with pytest.raises(ValueError):
            GqaAttention(*args, **bad)
