"""The mechanisms the Nipizen design brought, each alone against its plain function: attention with biases, norms over the whole
projection, a scaled rotation and a gate per value (every kernel that takes it, heads padded or not; inputs made so that ONE marked
key decides the last query, near, far and at page borders, in a prompt step and as a single token); the gated delta rule (sequences of
unequal length whose portions end anywhere in a chunk of four, shared q/k heads, up to 300 key channels, an input whose FIRST
token decides an output 250 tokens later, keys that come back); the mLSTM (gates below, at and far above the cap, both sides of the
denominator, a first token that counts for hundreds of steps); the pair with its scales; the experts with weighted inputs both
ways they run; rows cast out of wider rows."""
import numpy as np
import pytest
import torch

import plain_nipizen as P
from test_parts_gpu import Bench, close, load, rnd, run_mixer
from test_pirisun_parts_gpu import Ctx, f64

pytestmark = pytest.mark.gpu

DTYPES = [torch.float32, torch.bfloat16]


@pytest.fixture(scope="module")
def k():
    from zinfer_b200 import kernels
    kernels.require_cuda()
    return kernels


def np64(t):
    return {n: f64(a) for n, a in t.items()}


def in_portions(k, mixer, dtype, x, cuts, page=16):
    """`x` of one sequence fed in portions of the sizes `cuts`, in a slot that another sequence has used before."""
    bench = Bench(k, mixer, dtype, n_slots=2, max_seq=-(-max(256, x.shape[0]) // page) * page, page=page)
    slots = bench.cache.alloc_slots(2)
    ctx = bench.step(slots, [7, 9])
    mixer.forward(ctx, bench.call, rnd((16, x.shape[1]), 999, dtype).to(dtype).cuda(), torch.zeros((16, x.shape[1]), device="cuda"), False)
    bench.done(slots, [7, 9])
    bench.cache.free_slots(slots)
    slot = bench.cache.alloc_slots(2)[1:]
    got, at = [], 0
    for n in cuts:
        ctx = bench.step(slot, [n])
        out = torch.zeros((n, x.shape[1]), device="cuda")
        mixer.forward(ctx, bench.call, x[at:at + n].to(dtype).cuda(), out, False)
        bench.done(slot, [n])
        got.append(out.cpu())
        at += n
    assert at == x.shape[0]
    return torch.cat(got)


# ------------------------------------------------------------------------------- attention

def att_tensors(D, H, G, d, e, dtype, seed):
    t = {"q": rnd((H * d, D), seed, dtype, D ** -0.5), "k": rnd((G * d, D), seed + 1, dtype, D ** -0.5),
         "v": rnd((G * e, D), seed + 2, dtype, D ** -0.5), "o": rnd((D, H * e), seed + 3, dtype, (H * e) ** -0.5),
         "g": rnd((H * e, D), seed + 4, dtype, 2 * D ** -0.5), "q.norm": 1.0 + rnd((H * d,), seed + 5, dtype, 0.2),
         "k.norm": 1.0 + rnd((G * d,), seed + 6, dtype, 0.2)}
    for n, w in (("q.b", H * d), ("k.b", G * d), ("v.b", G * e)):
        t[n] = rnd((w,), seed + 7 + len(t), dtype, 0.5)
    return t


def make_att(D, H, G, d, e, scale, rot, t, dtype, pad=True, eps=1e-5):
    from zinfer_b200.parts import GqaAttention, RotaryEncoding
    position = None
    if rot:
        s = rot.get("scaling")
        position = RotaryEncoding(d, rot["base"], n_rot=rot["dims"], yarn=tuple(s[n] for n in ("factor", "original", "fast", "slow")) if s else None)
    return load(GqaAttention(D, H, G, d, "q", "k", "v", "o", q_norm_name="q.norm", k_norm_name="k.norm", norm_eps=eps, position=position,
                             scale=scale, value_dim=e, qk_norm_span="all", bias_names=("q.b", "k.b", "v.b", None), value_gate_name="g",
                             pad_heads=pad), t, dtype)


def plain_att(x, t, H, G, d, e, scale, rot, eps=1e-5):
    return P.attention(f64(x), np64(t), {"heads": H, "kv_heads": G, "dim": d, "vdim": e, "scale": scale, "rot": rot}, eps)


def rot_of(base, dims, scaling=None):
    r = {"base": base, "dims": dims}
    if scaling:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return r


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,H,G,d,e,scale,rot,page,pad", [
    (48, 4, 2, 16, 12, 0.6, rot_of(1000.0, 8, (4.0, 64, 8.0, 0.5)), 16, False), (64, 6, 6, 8, 16, 0.7, None, 16, False),
    (38, 5, 1, 10, 7, 0.6, rot_of(30.0, 10, (3.0, 20, 2.0, 0.3)), 64, True), (192, 6, 2, 64, 64, 0.25, rot_of(1e4, 64, (16.0, 256, 32.0, 1.0)), 64, True),
    (128, 4, 4, 96, 40, 0.2, rot_of(1e4, 96, (8.0, 100, 1.0, 1.0)), 64, True), (128, 2, 1, 128, 128, 0.15, rot_of(5e5, 64), 64, True),
    (64, 3, 1, 48, 64, 0.2, rot_of(3e3, 32, (2.0, 128, 4.0, 2.0)), 64, True), (32, 1, 1, 4, 6, 1.0, rot_of(20.0, 2), 16, False),
    (96, 2, 2, 160, 130, 0.1, rot_of(1e4, 160, (4.0, 512, 32.0, 1.0)), 16, True), (512, 12, 4, 64, 64, 0.3, rot_of(1e4, 64), 64, True)])
def test_attention_alone(k, dtype, D, H, G, d, e, scale, rot, page, pad):
    """Unequal sequences: a prompt step then single tokens, over several pages; the shapes include those of the tensor-core
    kernels, and heads padded up to them (whose norms count the padding)."""
    t = att_tensors(D, H, G, d, e, dtype, 40)
    mixer = make_att(D, H, G, d, e, scale, rot, t, dtype, pad)
    padded = pad and dtype == torch.bfloat16 and max(d, e) <= 128 and not (d == e and d in (64, 128))
    want = (d, e) if not padded else ((64, 64) if max(d, e) <= 64 else (128, 128))
    assert (mixer.run_head_dim, mixer.run_value_dim) == want
    xs = [rnd((n, D), 50 + b, dtype, 1.5) for b, n in enumerate((150, 40, 9))]
    outs = run_mixer(k, mixer, dtype, xs, [130, 17, 1], page=page)
    for b, x in enumerate(xs):
        close(outs[b], plain_att(x, t, H, G, d, e, scale, rot), dtype, f"sequence {b}")


def test_norm_epsilon_counts_in_padded_heads(k):
    """An epsilon as large as the mean square: scaled wrongly for the padding it would show."""
    D, H, G, d, e, rot = 64, 2, 2, 20, 30, rot_of(100.0, 20)
    t = att_tensors(D, H, G, d, e, torch.bfloat16, 45)
    x = rnd((70, D), 46, torch.bfloat16, 1.0)
    mixer = make_att(D, H, G, d, e, 0.5, rot, t, torch.bfloat16, eps=1.0)
    ref = plain_att(x, t, H, G, d, e, 0.5, rot, eps=1.0)
    assert np.abs(ref - plain_att(x, t, H, G, d, e, 0.5, rot, eps=64 / 20)).max() > 3e-2 * np.abs(ref).max()
    close(run_mixer(k, mixer, torch.bfloat16, [x], [50], page=64)[0], ref, torch.bfloat16, "epsilon")


T_MARK = 300


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,d,page", [(4, 2, 16, 16), (2, 1, 64, 64)])
@pytest.mark.parametrize("mark", [0, 1, 15, 16, 63, 64, 127, 255, 256, T_MARK - 2])
def test_one_marked_key_decides_the_last_query(k, dtype, H, G, d, page, mark):
    """Keys read the first third of the input, values the second, queries the last, through the keys' own matrix: the last token's
    query is made to match the key of token `mark` alone (a sharp scale, a rotation of two entries per head)."""
    D, T = 3 * d, T_MARK
    third = D // 3
    t = att_tensors(D, H, G, d, d, dtype, 70)
    t["k"].zero_()
    for g in range(G):           # an orthogonal map of inputs that are all 1 or -1; the two rotated entries of a head stay out of it
        t["k"][g * d:(g + 1) * d, :third] = torch.linalg.qr(t["k.norm"].new_tensor(np.random.default_rng(g).normal(size=(d, d))))[0].to(dtype).float()
        t["k"][g * d:g * d + 2] *= 0.125
    t["k.norm"][:], t["q.norm"][:] = 1.0, 1.0
    t["v"][:, :third] = 0.0
    t["v"][:, 2 * third:] = 0.0
    t["q"] = torch.zeros((H * d, D))
    t["q"][:, 2 * third:] = t["k"][:, :third].reshape(G, 1, d, third).expand(G, H // G, d, third).reshape(H * d, third)
    for n in ("q.b", "k.b"):
        t[n].zero_()
    rot, scale = rot_of(100.0, 2, (2.0, 50, 4.0, 1.0)), 30.0 / d
    mixer = make_att(D, H, G, d, d, scale, rot, t, dtype)
    x = rnd((T, D), 71, dtype)
    x[:, :third] = torch.sign(x[:, :third])
    x[:, 2 * third:] = torch.sign(x[:, 2 * third:])
    x[T - 1, 2 * third:] = x[mark, :third]
    ref = plain_att(x, t, H, G, d, d, scale, rot)
    other = x.clone()
    other[mark, third:2 * third] = rnd((third,), 72, dtype)
    moved = plain_att(other, t, H, G, d, d, scale, rot)
    assert np.abs(ref[-1] - moved[-1]).max() > 0.05 * np.abs(ref).max(), "the marked key does not decide the last query"
    for prompt in (T, T - 1, 200):
        close(run_mixer(k, mixer, dtype, [x], [prompt], page=page)[0], ref, dtype, f"prompt of {prompt}")


@pytest.mark.parametrize("rows", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("gate", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,width,valid,skip", [(4, 64, 64, 96), (3, 128, 80, 104), (5, 7, 7, 3)])
def test_gate_per_value_in_either_dtype(k, rows, gate, H, width, valid, skip):
    r, g = rnd((11, H * width), 1, rows), rnd((11, skip + H * valid), 2, gate, 2.0)
    ref = f64(r).reshape(11, H, width).copy()
    ref[:, :, :valid] *= P.sigmoid(f64(g)[:, skip:].reshape(11, H, valid))
    close(k.value_gate(r.to(rows).cuda(), g.to(gate).cuda()[:, skip:], H, valid), ref.reshape(11, -1), rows, "gate per value")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("n,d", [(3, 64), (300, 64), (300, 48)])
def test_rotation_amplitude_in_per_head_preparation(k, dtype, n, d):
    """The factor on cosines and sines in the kernels that prepare heads one by one (and a token at a time), without norms."""
    from zinfer_b200.parts import GqaAttention, RotaryEncoding
    D, H, G = 64, 4, 2
    t = {x: a for x, a in att_tensors(D, H, G, d, d, dtype, 80).items() if x in "qkvo"}
    rot = rot_of(500.0, d, (6.0, 64, 8.0, 0.5))
    mixer = load(GqaAttention(D, H, G, d, "q", "k", "v", "o", position=RotaryEncoding(d, 500.0, yarn=(6.0, 64, 8.0, 0.5)), scale=0.05), t, dtype)
    x = rnd((n, D), 81, dtype, 1.5)
    freq, amp = P.rotation(rot)
    q, kk = (P.rotate((f64(x) @ f64(t[w]).T).reshape(n, h, d), freq, amp) for w, h in (("q", H), ("k", G)))
    v = (f64(x) @ f64(t["v"]).T).reshape(n, G, d)
    out = np.zeros((n, H, d))
    for i in range(n):
        for a in range(H):
            sc = (kk[:i + 1, a // 2] @ q[i, a]) * 0.05
            w = np.exp(sc - sc.max())
            out[i, a] = w / w.sum() @ v[:i + 1, a // 2]
    close(run_mixer(k, mixer, dtype, [x], [n - 1], page=64)[0], out.reshape(n, -1) @ f64(t["o"]).T, dtype, "amplitude")


# ------------------------------------------------------------------------------- gated delta rule

def delta_tensors(D, H, G, d, e, taps, ra, rg, dtype, seed):
    t = {"q": rnd((G * d, D), seed, dtype, D ** -0.5), "k": rnd((G * d, D), seed + 1, dtype, D ** -0.5), "v": rnd((H * e, D), seed + 2, dtype, D ** -0.5),
         "b": rnd((H, D), seed + 3, dtype, 2 * D ** -0.5), "A_log": rnd((H,), seed + 4, dtype, 1.0) - 2.0, "a1": rnd((ra, D), seed + 5, dtype, D ** -0.5),
         "a2": rnd((H * d, ra), seed + 6, dtype, 2 * ra ** -0.5), "dt_bias": rnd((H * d,), seed + 7, dtype, 1.0), "g1": rnd((rg, D), seed + 8, dtype, D ** -0.5),
         "g2": rnd((H * e, rg), seed + 9, dtype, 2 * rg ** -0.5), "norm": 1.0 + rnd((e,), seed + 10, dtype, 0.2), "o": rnd((D, H * e), seed + 11, dtype, (H * e) ** -0.5)}
    for i, (n, w) in enumerate((("q", G * d), ("k", G * d), ("v", H * e))):
        t[n + ".conv"] = rnd((w, taps), seed + 12 + i, dtype, 0.7)
        t[n + ".conv"][:, -1] += 1.0
    return t


def make_delta(D, H, G, d, e, taps, t, dtype, eps=1e-5):
    from zinfer_b200.parts import GatedDelta
    return load(GatedDelta(D, H, G, d, e, taps, "q", "k", "v", "q.conv", "k.conv", "v.conv", "b", "A_log", "a1", "a2", "dt_bias", "g1", "g2",
                           "norm", "o", norm_eps=eps), t, dtype)


def plain_delta(x, t, H, G, d, e, eps=1e-5):
    return P.delta_mixer(f64(x), np64(t), {"heads": H, "kv_heads": G, "dim": d, "vdim": e}, eps)


DELTA_SHAPES = [(48, 4, 2, 12, 10, 3, 6, 9), (32, 1, 1, 4, 4, 1, 1, 1), (128, 4, 4, 32, 64, 4, 32, 24), (38, 2, 2, 7, 5, 5, 7, 4),
                (64, 3, 1, 64, 20, 2, 16, 8), (128, 2, 2, 128, 72, 4, 40, 24), (64, 6, 3, 100, 33, 4, 20, 12), (64, 2, 1, 200, 24, 4, 8, 8),
                (64, 1, 1, 300, 9, 3, 8, 16)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,H,G,d,e,taps,ra,rg", DELTA_SHAPES)
def test_delta_rule_alone(k, dtype, D, H, G, d, e, taps, ra, rg):
    """Sequences of unequal length in one batch, whose prompts end with one to four tokens in their last chunk, then single tokens."""
    t = delta_tensors(D, H, G, d, e, taps, ra, rg, dtype, 10)
    mixer = make_delta(D, H, G, d, e, taps, t, dtype)
    xs = [rnd((n, D), 20 + b, dtype) for b, n in enumerate((90, 37, 26, 12))]
    outs = run_mixer(k, mixer, dtype, xs, [70, 17, 23, 4], page=16)
    for b, x in enumerate(xs):
        close(outs[b], plain_delta(x, t, H, G, d, e), dtype, f"sequence {b}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [(1, 1, 1, 1, 60), (2, 2, 2, 58), (3, 5, 7, 2, 47), (64,), (9, 1, 8, 2, 44), (40, 2, 1, 1, 20)])
@pytest.mark.parametrize("shape", [DELTA_SHAPES[2], DELTA_SHAPES[3]])
def test_delta_rule_in_portions(k, dtype, shape, cuts):
    """Portions down to one token, in a slot used before: the convolution's last inputs and the matrices pass from one to the next."""
    D, H, G, d, e, taps, ra, rg = shape
    t = delta_tensors(*shape, dtype, 30)
    x = rnd((64, D), 31, dtype)
    close(in_portions(k, make_delta(D, H, G, d, e, taps, t, dtype), dtype, x, cuts), plain_delta(x, t, H, G, d, e), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [260, 101, 2, 1])
def test_delta_rule_keeps_the_first_token_for_hundreds_of_steps(k, dtype, prompt):
    """Later keys are made tiny (their share of the unit vector's epsilon), decays lie next to 1: every output is the first
    tokens' write; a state that is lost, zeroed or decayed wrongly changes everything."""
    D, H, G, d, e, taps = 32, 2, 1, 8, 8, 2
    t = delta_tensors(D, H, G, d, e, taps, 4, 4, dtype, 40)
    t["k"][:, D // 2:] = 0.0                        # keys read the first half of the input only
    t["q"][:, :D // 2] = 0.0
    t["v"][:, :D // 2] = 0.0
    t["a2"].zero_()
    t["dt_bias"][:], t["A_log"][:] = -4.0, -3.0
    mixer = make_delta(D, H, G, d, e, taps, t, dtype, eps=1e-8)
    x = rnd((260, D), 41, dtype)
    x[1:, :D // 2] *= 2.0 ** -14
    ref = plain_delta(x, t, H, G, d, e, eps=1e-8)
    without = x.clone()
    without[0, D // 2:] = -x[0, D // 2:]
    assert np.abs(ref[-1] - plain_delta(without, t, H, G, d, e, eps=1e-8)[-1]).max() > 0.1 * np.abs(ref).max()
    close(run_mixer(k, mixer, dtype, [x], [prompt], page=16)[0], ref, dtype, f"prompt of {prompt}")


def test_delta_rule_replaces_what_a_returning_key_reads(k):
    """Four keys come round again and again without decay and with beta next to 1: the read must see the writes of the same
    chunk (one to three tokens before) and of chunks before."""
    D, H, G, d, e, taps, dtype = 32, 2, 2, 8, 6, 1, torch.float32
    t = delta_tensors(D, H, G, d, e, taps, 4, 4, dtype, 50)
    t["k"][:, D // 2:] = 0.0
    t["q"] = t["k"].clone()
    t["k.conv"][:] = t["q.conv"][:] = 1.0
    t["a2"].zero_()
    t["dt_bias"][:] = -12.0
    t["b"][:, D // 2:] = 0.0
    keys = rnd((4, D // 2), 51, dtype, 2.0)
    t["b"][:, :D // 2] = 6.0 * (torch.linalg.pinv(keys) @ torch.ones(4))[None]      # every key's beta logit is 6
    for order in ([0, 1, 2, 3], [0, 0, 1, 0, 2, 1], [3, 3, 3, 3, 3]):
        x = rnd((61, D), 52, dtype)
        for i in range(61):
            x[i, :D // 2] = keys[order[i % len(order)]]
        ref = plain_delta(x, t, H, G, d, e)
        for prompt in (61, 30, 1):
            close(run_mixer(k, make_delta(D, H, G, d, e, taps, t, dtype), dtype, [x], [prompt], page=16)[0], ref, dtype, f"{order} {prompt}")


@pytest.mark.parametrize("lanes", [8, 16])
def test_delta_rule_in_either_layout(k, lanes):
    D, H, G, d, e, taps = 64, 3, 3, 112, 50, 3
    t = delta_tensors(D, H, G, d, e, taps, 8, 8, torch.float32, 60)
    x = rnd((75, D), 61, torch.float32)
    k.delta_force_lanes(lanes)
    try:
        outs = run_mixer(k, make_delta(D, H, G, d, e, taps, t, torch.float32), torch.float32, [x], [70], page=16)
    finally:
        k.delta_force_lanes(0)
    close(outs[0], plain_delta(x, t, H, G, d, e), torch.float32, f"{lanes} lanes")


# ------------------------------------------------------------------------------- mLSTM

def mem_tensors(D, H, d, e, dtype, seed, gate=3.0):
    return {"q": rnd((H * d, D), seed, dtype, D ** -0.5), "k": rnd((H * d, D), seed + 1, dtype, D ** -0.5), "v": rnd((H * e, D), seed + 2, dtype, D ** -0.5),
            "g": rnd((H * e, D), seed + 3, dtype, D ** -0.5), "i": rnd((H, D), seed + 4, dtype, gate * D ** -0.5), "f": rnd((H, D), seed + 5, dtype, gate * D ** -0.5),
            "i.b": rnd((H,), seed + 6, dtype, 1.0) - 1.0, "f.b": rnd((H,), seed + 7, dtype, 1.0) + 3.0, "norm": 1.0 + rnd((H * e,), seed + 8, dtype, 0.2),
            "o": rnd((D, H * e), seed + 9, dtype, (H * e) ** -0.5)}


def make_mem(D, H, d, e, cap, t, dtype, eps=1e-5):
    from zinfer_b200.parts import MLstm
    return load(MLstm(D, H, d, e, cap, "q", "k", "v", "i", "i.b", "f", "f.b", "g", "norm", "o", norm_eps=eps), t, dtype)


def plain_mem(x, t, H, d, e, cap, eps=1e-5):
    return P.mlstm(f64(x), np64(t), {"heads": H, "dim": d, "vdim": e, "gate_cap": cap}, eps)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,H,d,e,cap,gate", [(48, 3, 8, 10, 5.0, 3.0), (64, 2, 16, 8, 2.0, 6.0), (128, 4, 32, 64, 15.0, 3.0), (38, 2, 6, 5, 1.0, 3.0),
                                              (64, 1, 4, 31, 30.0, 20.0), (64, 2, 160, 32, 10.0, 1.0), (64, 1, 300, 33, 3.0, 3.0), (64, 2, 1, 1, 4.0, 3.0)])
def test_mlstm_alone(k, dtype, D, H, d, e, cap, gate):
    """Unequal sequences, prompts then single tokens.  The widths put the normaliser's column alone into a block of columns
    (32 values), last in one (31) and in the middle; the gates reach below, at and far above the cap."""
    t = mem_tensors(D, H, d, e, dtype, 10, gate)
    mixer = make_mem(D, H, d, e, cap, t, dtype)
    xs = [rnd((n, D), 20 + b, dtype) for b, n in enumerate((90, 37, 12))]
    outs = run_mixer(k, mixer, dtype, xs, [70, 17, 1], page=16)
    for b, x in enumerate(xs):
        close(outs[b], plain_mem(x, t, H, d, e, cap), dtype, f"sequence {b}")


def test_mlstm_both_sides_of_the_denominator(k):
    """The oracle's own denominators: inputs for which |n . q| decides at some tokens and exp(-m) at others."""
    D, H, d, e, cap = 48, 3, 8, 10, 5.0
    t = np64(mem_tensors(D, H, d, e, torch.float32, 10, 3.0))
    h = f64(rnd((90, D), 20, torch.float32))
    q, kk = (h @ t["q"].T).reshape(90, H, d) * d ** -0.5, (h @ t["k"].T).reshape(90, H, d)
    i, f = cap * np.tanh((h @ t["i"].T + t["i.b"]) / cap), P.log_sigmoid(cap * np.tanh((h @ t["f"].T + t["f.b"]) / cap))
    sides = []
    for a in range(H):
        z, m = np.zeros(d), 0.0
        for s in range(90):
            m, old = max(f[s, a] + m, i[s, a]), m
            z = np.exp(f[s, a] + old - m) * z + np.exp(i[s, a] - m) * kk[s, a]
            sides.append(abs(z @ q[s, a]) > np.exp(-m))
    assert 0.1 < np.mean(sides) < 0.9


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cuts", [(1, 1, 1, 61), (2, 2, 60), (15, 16, 17, 16), (16, 48), (64,), (33, 2, 29)])
def test_mlstm_in_portions(k, dtype, cuts):
    """Portions whose ends lie inside, at and just behind the groups of tokens the kernel stages at once."""
    D, H, d, e, cap = 64, 2, 24, 40, 6.0
    t = mem_tensors(D, H, d, e, dtype, 30)
    x = rnd((64, D), 31, dtype)
    close(in_portions(k, make_mem(D, H, d, e, cap, t, dtype), dtype, x, cuts), plain_mem(x, t, H, d, e, cap), dtype, f"{cuts}")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("prompt", [260, 100, 2, 1])
def test_mlstm_keeps_the_first_token_for_hundreds_of_steps(k, dtype, prompt):
    """The first token's input gate stands high above all later ones and the forget gates next to 1: every output is the first
    token's value, and a running maximum that is lost or starts at anything but 0 shows."""
    D, H, d, e, cap = 32, 2, 8, 8, 12.0
    t = mem_tensors(D, H, d, e, dtype, 40)
    t["i"][:] = 0.0
    t["i"][:, 0] = 4.0
    t["f"][:] = 0.0
    t["f.b"][:], t["i.b"][:] = 9.0, -2.0
    x = rnd((260, D), 41, dtype)
    x[:, 0] = -1.0
    x[0, 0] = 2.0
    ref = plain_mem(x, t, H, d, e, cap)
    other = x.clone()
    other[0, 1:] = rnd((D - 1,), 42, dtype)
    assert np.abs(ref[-1] - plain_mem(other, t, H, d, e, cap)[-1]).max() > 0.1 * np.abs(ref).max()
    got = run_mixer(k, make_mem(D, H, d, e, cap, t, dtype), dtype, [x], [prompt], page=16)[0]
    # where a query all but misses the first key its two products are small differences of larger terms: 1e-4 in 32-bit
    assert np.abs(f64(got) - ref).max() <= (1e-4 if dtype == torch.float32 else 1.5e-2) * np.abs(ref).max()


# ------------------------------------------------------------------------------- the pair

@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,left,right,scales,page", [
    (48, (4, 2, 16, 12, 0.3, rot_of(1000.0, 8, (4.0, 64, 8.0, 0.5))), (4, 2, 12, 10, 3, 6, 9), (0.7, -0.9), 16),
    (256, (6, 2, 64, 64, 0.2, rot_of(1e4, 64)), (4, 4, 32, 64, 4, 32, 24), (0.3, 1.4), 64)])
def test_pair_with_scales(k, dtype, D, left, right, scales, page):
    """a * A(h) + b * B(h), through prompt steps (more rows than the few-row contractions take) and single-token steps."""
    from zinfer_b200.parts import MixerPair
    H, G, d, e, scale, rot = left
    Hr, Gr, dr, er, taps, ra, rg = right
    tl, tr = att_tensors(D, H, G, d, e, dtype, 80), delta_tensors(D, Hr, Gr, dr, er, taps, ra, rg, dtype, 110)
    a, b = make_att(D, H, G, d, e, scale, rot, tl, dtype), make_delta(D, Hr, Gr, dr, er, taps, tr, dtype)
    pair = MixerPair(D, a, b, scales=scales)
    pair.load({}, dtype, torch.device("cuda"))
    assert pair.weight_specs() == [] and pair.kv_request() == a.kv_request() and pair.state_request() == b.state_request()
    xs = [rnd((n, D), 100 + i, dtype) for i, n in enumerate((100, 30, 5))]
    outs = run_mixer(k, pair, dtype, xs, [90, 17, 1], page=page)
    for i, x in enumerate(xs):
        ref = scales[0] * plain_att(x, tl, H, G, d, e, scale, rot) + scales[1] * plain_delta(x, tr, Hr, Gr, dr, er)
        close(outs[i], ref, dtype, f"sequence {i}")


# ------------------------------------------------------------------------------- experts

def expert_tensors(D, F, E, dtype, seed):
    t = {"router": rnd((E, D), seed, torch.bfloat16, 3.0 * D ** -0.5)}
    for e in range(E):
        t[f"e{e}.up"], t[f"e{e}.down"] = rnd((F, D), seed + 2 * e + 1, dtype, 1.5 * D ** -0.5), rnd((D, F), seed + 2 * e + 2, dtype, F ** -0.5)
    return t


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("D,F,E,top,rows", [(48, 24, 6, 2, 7), (64, 72, 3, 3, 33), (128, 64, 8, 2, 300), (128, 256, 8, 3, 200), (38, 10, 5, 2, 130),
                                            (256, 96, 12, 1, 3), (128, 512, 4, 4, 700), (64, 40, 1, 1, 120), (64, 16, 40, 5, 515)])
def test_ungated_experts_with_weighted_inputs(k, dtype, D, F, E, top, rows):
    """The streaming kernels (few rows, single-token steps) and the grouped contractions (many rows; hidden widths that are and are
    not whole tiles) against the plain function; ids and weights against the plain choice.  Rows whose choice is a close call are left out
    of the bfloat16 comparison (they are independent of one another)."""
    from zinfer_b200.parts import RoutedMoE
    t = expert_tensors(D, F, E, dtype, 20)
    ff = load(RoutedMoE(D, F, E, top, "router", lambda e: (f"e{e}.up", f"e{e}.down"), score="sigmoid", renormalize=False, weight_input=True,
                        act="relu_squared"), t, dtype)
    x = rnd((rows, D), 5, dtype)
    W = np64(t)
    margins = [np.inf] * rows
    ref = P.moe(f64(x), W, {"experts": E, "top": top}, margins)
    keep = np.array([m > (0.01 if dtype == torch.bfloat16 else 1e-6) for m in margins])
    assert keep.sum() >= max(1, rows // 3)
    ids, wts = k.moe_router(x.to(dtype).cuda(), ff.w_router, top, sigmoid=True, renormalize=False)
    s = P.sigmoid(f64(x) @ W["router"].T)
    for i in np.flatnonzero(keep)[:40]:
        chosen = sorted(range(E), key=lambda e: (-s[i, e], e))[:top]
        assert ids[i].tolist() == chosen or dtype == torch.bfloat16 and set(ids[i].tolist()) == set(chosen)
        assert np.allclose(wts[i].cpu().numpy(), s[i, ids[i].tolist()], rtol=1e-4, atol=1e-6)
    sel = torch.from_numpy(keep).cuda()
    outs = {}
    for decode in (False, True):
        out = torch.full((rows, D), 0.5, device="cuda")
        ff.forward(Ctx(k, dtype, rows, decode), x.to(dtype).cuda(), out, True)
        outs[decode] = out - 0.5
        close(outs[decode][sel], ref[keep], dtype, "decode" if decode else "prompt")
    i = int(np.flatnonzero(keep)[-1])
    alone = torch.zeros((1, D), device="cuda")
    ff.forward(Ctx(k, dtype, 1, True), x[i:i + 1].to(dtype).cuda(), alone, False)
    assert torch.allclose(alone[0], outs[True][i], atol=2e-6 * float(outs[True][i].abs().max()) + 1e-6)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("act", ["gelu_tanh", "silu", "relu"])
@pytest.mark.parametrize("rows", [5, 150])
def test_a_weight_on_the_input_is_not_one_on_the_output(k, dtype, act, rows):
    """Activations that are no power of their input tell the two apart; softmax scores, renormalised, go with it too."""
    from zinfer_b200.parts import RoutedMoE
    D, F, E, top = 64, 48, 3, 3
    t = expert_tensors(D, F, E, dtype, 30)
    ff = load(RoutedMoE(D, F, E, top, "router", lambda e: (f"e{e}.up", f"e{e}.down"), weight_input=True, act=act), t, dtype)
    x = rnd((rows, D), 31, dtype, 2.0)
    z = f64(x) @ f64(t["router"]).T
    s = np.exp(z - z.max(1, keepdims=True))
    s /= s.sum(1, keepdims=True)
    fn = {"relu": lambda u: np.maximum(u, 0), "silu": lambda u: u * P.sigmoid(u),
          "gelu_tanh": lambda u: 0.5 * u * (1 + np.tanh(np.sqrt(2 / np.pi) * (u + 0.044715 * u ** 3)))}[act]
    ref = sum(fn((s[:, e:e + 1] * f64(x)) @ f64(t[f"e{e}.up"]).T) @ f64(t[f"e{e}.down"]).T for e in range(E))
    for decode in (False, True):
        out = torch.zeros((rows, D), device="cuda")
        ff.forward(Ctx(k, dtype, rows, decode), x.to(dtype).cuda(), out, False)
        close(out, ref, dtype, f"{act} {'decode' if decode else 'prompt'}")


@pytest.mark.parametrize("rows,width,ld,at", [(7, 24, 40, 8), (130, 33, 70, 5), (1, 16, 16, 0), (5, 8, 1000, 4)])
def test_cast_of_columns(k, rows, width, ld, at):
    x = rnd((rows, ld), 1, torch.float32).cuda()
    got = k.cast_rows(x[:, at:at + width], torch.bfloat16)
    assert got.is_contiguous() and torch.equal(got, x[:, at:at + width].to(torch.bfloat16))
