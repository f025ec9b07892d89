"""The Demavik design in the engine against the plain implementation in ``plain_demavik``.

First each mechanism's kernels alone (the short convolution; the selective scan in portions, token by token
and in chunks side by side, with its state; gated linear attention in chunks and token by token; the norm over a
whole projection with rotation and cache writes; the pair embedding; the softmax router; float32 sums that join
behind a norm), then whole models through trace replay: whole prompts, the last tokens decoded one by one,
portions down to two tokens, mixed batches in a pool so small that pages and slots are used again, long
decoding, long prompts, the first tokens, a key far away and at page borders (of the layer's own and of the
layer whose keys it reads), writes that are recalled hundreds of tokens later, the edges of the convolution and
of the pair embedding, and greedy generation through the engine's entry point and scheduler.
"""
import numpy as np
import pytest
import torch

import demavik_configs as dc
import plain_demavik as plain
from helpers import check_logits as _check_logits, random_prompts

pytestmark = pytest.mark.gpu

DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}
# A router whose choice is closer than this in the plain model may choose otherwise in bfloat16.
CLEAR = 0.06


def check_logits(got, want, dtype, what, clear=None):
    """float32 is the sharp test, row by row.  In bfloat16 the rows whose router had a close call (``clear``
    false) are left out; of the others one in fifty (one at least) may miss the tolerance by up to a
    factor of four, and one in five hundred by up to eight: a close call of an earlier token reaches later ones
    through states and keys, and where a sublayer's result nearly cancels, the division by its root mean square
    multiplies the rounding."""
    want = torch.from_numpy(np.asarray(want))
    if dtype == "float32":
        _check_logits(got, want, dtype, what, f32_tolerance=4e-5)
        return
    got = np.asarray(got)
    assert np.isfinite(got).all(), f"{what}: logits are not finite"
    if clear is not None:
        if not clear.any():
            return
        got, want = got[clear], want[torch.from_numpy(clear)]
    got_t = torch.from_numpy(np.ascontiguousarray(got)).double()
    ratio = (got_t - want.double()).abs().amax(-1) / want.double().abs().amax(-1).clamp_min(1e-3)
    loose = ratio > 6e-2
    assert int(loose.sum()) <= max(1, len(ratio) // 50), f"{what}: {int(loose.sum())} of {len(ratio)} rows miss the tolerance"
    far = ratio > 0.24
    assert int(far.sum()) <= len(ratio) // 500 and float(ratio.max()) <= 0.5, (
        f"{what}: row {int(ratio.argmax())} is off by {float(ratio.max()):.3f} of its largest logit")
    keep = ~loose
    if int(keep.sum()):
        _check_logits(got[keep.numpy()], want[keep], dtype, what, bf16_tolerance=6e-2, bf16_min_cosine=0.997)


def close(got, want, dtype, what, scale=None, f32=4e-6, bf16=1.2e-2):
    got = got.double().cpu()
    want = torch.as_tensor(np.asarray(want)).double()
    scale = float(want.abs().max()) if scale is None else scale
    tol = (f32 if dtype == "float32" else bf16) * max(scale, 1e-6)
    err = float((got - want).abs().max())
    assert err <= tol, f"{what} ({dtype}): max error {err:.3e}, allowed {tol:.3e}"


def dev_int(a):
    return torch.tensor(np.asarray(a, dtype=np.int32)).cuda()


def num(t):
    return t.double().cpu().numpy()


class Steps:
    """Steps of a few sequences: step i takes ``cuts[s][i]`` tokens of every sequence s that has so many cuts."""

    def __init__(self, lengths, cuts, slots):
        self.lengths, self.cuts, self.slots = lengths, cuts, slots
        assert all(sum(c) == n for c, n in zip(cuts, lengths))

    def __iter__(self):
        done = [0] * len(self.lengths)
        for step in range(max(len(c) for c in self.cuts)):
            live = [s for s in range(len(self.cuts)) if step < len(self.cuts[s])]
            sizes = [self.cuts[s][step] for s in live]
            spans = [(s, done[s], done[s] + n) for s, n in zip(live, sizes)]
            starts = np.concatenate([[0], np.cumsum(sizes)[:-1]])
            yield spans, sum(sizes), dev_int(starts), dev_int(sizes), dev_int([self.slots[s] for s in live])
            for s, n in zip(live, sizes):
                done[s] += n


def take(parts, spans):
    return torch.cat([parts[s][a:b] for s, a, b in spans]).cuda()


def give(got, spans, rows):
    at = 0
    for s, a, b in spans:
        got[s][a:b] = num(rows[at : at + b - a])
        at += b - a


CUTS = [[1, 1, 2, 17, 1, 1, 20, 2, 1, 1, 1, 1], [1, 2, 1, 10, 1, 1, 4], [3, 1, 1, 1, 1, 1, 2, 1]]
LENGTHS = [49, 20, 11]


# ------------------------------------------------------------------------------------ kernels
@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("channels,taps", [(64, 4), (40, 3), (24, 2), (16, 1), (13, 4), (9, 5), (72, 9), (8, 40)])
def test_convolution_in_portions(dtype, channels, taps):
    """Portions down to one token (shorter than the taps too) beside each other; every sequence has its own state row,
    others stay as they are.  More taps than a tile of tokens holds run as one tile."""
    from velox_b200.ops import kernels as k

    dt = DTYPES[dtype]
    gen = torch.Generator().manual_seed(channels + taps)
    w, b = 0.6 * torch.randn(channels, taps, generator=gen), 0.5 * torch.randn(channels, generator=gen)
    x = [torch.randn(n, channels, generator=gen).to(dt) for n in LENGTHS]
    want = [plain.silu(plain.causal_conv(num(v), num(w), num(b))) for v in x]
    state = torch.zeros(6, max((taps - 1) * channels, 1)).cuda()
    state[[1, 2, 4]] = 7.0
    got = [np.zeros(v.shape) for v in want]
    for spans, T, q_start, q_len, slots in Steps(LENGTHS, CUTS, [3, 0, 5]):
        wide = torch.cat([torch.zeros(T, 8, dtype=dt).cuda(), take(x, spans)], dim=1)
        out = torch.full((T, channels), 9.0, dtype=dt).cuda()
        k.conv_act(wide[:, 8:], w.t().contiguous().cuda(), b.cuda(), state, out, q_start, q_len, slots, len(spans), T, k.ACT_SILU)
        give(got, spans, out)
    for s in range(3):
        close(torch.from_numpy(got[s]), want[s], dtype, f"sequence {s}")
    assert bool((state[[1, 2, 4]] == 7.0).all()), "another slot's state has changed"


class ScanCase:
    def __init__(self, dtype, inner, N, rank, lengths, seed, memory=0.0):
        from velox_b200.ops import kernels

        self.k, self.dt, self.dtype = kernels, DTYPES[dtype], dtype
        self.inner, self.N, self.rank, self.lengths = inner, N, rank, lengths
        gen = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=gen)
        self.a_log, self.bias, self.d = -0.5 + 0.8 * rand(inner, N), -1.5 - memory + rand(inner), rand(inner)
        self.w_dt = (rand(inner, rank) / rank ** 0.5).to(self.dt)
        self.x, self.z = [[rand(n, inner).to(self.dt) for n in lengths] for _ in range(2)]
        self.low = [rand(n, rank + 2 * N).to(self.dt) for n in lengths]
        self.start = [torch.zeros(inner, N) for _ in lengths]

    def plain(self):
        outs, states = [], []
        for s in range(len(self.lengths)):
            low = num(self.low[s])
            dt = plain.softplus(low[:, : self.rank] @ num(self.w_dt).T + num(self.bias))
            y, S = plain.selective_scan(num(self.x[s]), dt, -np.exp(num(self.a_log)), low[:, self.rank : self.rank + self.N],
                                        low[:, self.rank + self.N :], num(self.d), S=num(self.start[s]))
            outs.append(y * plain.silu(num(self.z[s])))
            states.append(S)
        return outs, states

    def run(self, cuts, slots, num_slots, chunk=0, step_kernel=True):
        k, I, N, R = self.k, self.inner, self.N, self.rank
        state = torch.zeros(num_slots, -(-I * N // 4) * 4).cuda()
        spare = [i for i in range(num_slots) if i not in slots]
        for s, slot in enumerate(slots):
            state[slot, : I * N] = self.start[s].reshape(-1).cuda()
        state[spare] = 7.0
        a2 = (-torch.exp(self.a_log.double()) * np.log2(np.e)).float().contiguous().cuda()
        bias, d, w_dt = self.bias.cuda(), self.d.cuda(), self.w_dt.contiguous().cuda()
        status = torch.zeros(4, dtype=torch.int32).cuda()
        got = [np.zeros((n, I)) for n in self.lengths]
        for spans, T, q_start, q_len, seq_slots in Steps(self.lengths, cuts, slots):
            x, z, low = take(self.x, spans), take(self.z, spans), take(self.low, spans)
            xz = torch.cat([x, z], dim=1)
            out = torch.zeros(T, I, dtype=self.dt).cuda()
            if step_kernel and all(b - a == 1 for _, a, b in spans):
                assert k.selective_step(xz[:, :I], low, w_dt, bias, a2, d, xz[:, I:], out, state, q_start, seq_slots, len(spans))
            else:
                dt = low[:, :R].float() @ w_dt.float().T
                scratch = {}
                if chunk:
                    places = T // chunk + len(spans) + 1
                    scratch = dict(chunk=chunk, chunk_states=torch.full((places * I * N,), np.nan).cuda(),
                                   chunk_dt=torch.full((places * I,), np.nan).cuda())
                k.selective_scan(xz[:, :I], dt, bias, a2, low[:, R:], d, xz[:, I:], out, state, q_start, q_len, seq_slots,
                                 len(spans), T, status, **scratch)
            give(got, spans, out)
        assert int(status[0]) == 0
        assert bool((state[spare] == 7.0).all()), "another slot's state has changed"
        return got, [num(state[slot, : I * N].view(I, N)) for slot in slots]


SCAN_SIZES = [(96, 12, 6), (64, 16, 8), (54, 5, 3), (40, 1, 1), (33, 4, 2), (130, 24, 16), (40, 40, 5), (24, 130, 2), (8, 300, 24),
              (300, 8, 160)]


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("inner,N,rank", SCAN_SIZES)
def test_selective_scan_in_portions(dtype, inner, N, rank):
    """Three sequences side by side in portions down to one token, steps of single tokens (their own kernel) among
    them, from states that are not zero."""
    case = ScanCase(dtype, inner, N, rank, LENGTHS, seed=inner + N)
    gen = torch.Generator().manual_seed(4)
    case.start = [torch.randn(s.shape, generator=gen) for s in case.start]
    want, want_state = case.plain()
    got, state = case.run(CUTS, slots=[3, 0, 5], num_slots=6)
    for s in range(3):
        close(torch.from_numpy(got[s]), want[s], dtype, f"sequence {s}", f32=1e-5)
        close(torch.from_numpy(state[s]), want_state[s], "float32", f"state of sequence {s}", f32=1e-5)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("inner,N,chunk", [(40, 16, 64), (24, 6, 80), (130, 3, 64), (20, 70, 96)])
def test_selective_scan_in_chunks(dtype, inner, N, chunk):
    """Long portions in chunks side by side: many chunks and a bit, whole chunks, a short portion and a single token in
    one step, from states that are not zero and with step sizes so small that every chunk's start matters."""
    first, second, third = [400, 2 * chunk, 37, 1], [3, 200, 1, 20], [1, 1, 1, 1]
    lengths = [a + b + c for a, b, c in zip(first, second, third)]
    case = ScanCase(dtype, inner, N, 4, lengths, seed=inner, memory=4.0)
    gen = torch.Generator().manual_seed(3)
    case.start = [torch.randn(s.shape, generator=gen) for s in case.start]
    want, want_state = case.plain()
    got, state = case.run([list(c) for c in zip(first, second, third)], slots=[0, 2, 1, 3], num_slots=5, chunk=chunk)
    for s in range(4):
        close(torch.from_numpy(got[s]), want[s], dtype, f"sequence {s}", f32=2e-5)
        close(torch.from_numpy(state[s]), want_state[s], "float32", f"state of sequence {s}", f32=2e-5)


def test_step_sizes_from_nothing_to_everything():
    """Logits from -30 (a step of nothing: the state stays) to 60 (it forgets everything), in both kernels and dtypes."""
    for dtype in DTYPES:
        case = ScanCase(dtype, 32, 8, 1, [31], seed=1)
        case.w_dt = torch.ones(32, 1).to(case.dt)
        case.bias = torch.zeros(32)
        case.low[0][:, 0] = torch.linspace(-30.0, 60.0, 31).to(case.dt)
        case.start = [torch.ones(32, 8)]
        want, want_state = case.plain()
        for cuts in ([31], [1] * 31):
            got, state = case.run([cuts], slots=[0], num_slots=1)
            close(torch.from_numpy(got[0]), want[0], dtype, "outputs", f32=2e-6)
            close(torch.from_numpy(state[0]), want_state[0], "float32", "state", f32=2e-6)


class LinearCase:
    def __init__(self, dtype, heads, dim, vdim, tau, rank, lengths, seed, memory=0.0):
        from velox_b200.ops import kernels

        self.k, self.dt, self.dtype = kernels, DTYPES[dtype], dtype
        self.H, self.D, self.V, self.tau, self.rank, self.lengths = heads, dim, vdim, tau, rank, lengths
        gen = torch.Generator().manual_seed(seed)
        rand = lambda *s: torch.randn(*s, generator=gen)
        keys, inner = heads * dim, heads * vdim
        self.q, self.kk = [[rand(n, keys).to(self.dt) for n in lengths] for _ in range(2)]
        self.v, self.g = [[rand(n, inner).to(self.dt) for n in lengths] for _ in range(2)]
        self.low = [rand(n, rank).to(self.dt) for n in lengths]
        self.a_up = (1.5 * rand(keys, rank) / rank ** 0.5).to(self.dt)
        self.bias = 1.0 + memory + rand(keys)
        self.norm, self.eps = 1.0 + 0.3 * rand(vdim), 1e-5
        self.start = [torch.zeros(heads, dim, vdim) for _ in lengths]

    def plain(self):
        H, D, V = self.H, self.D, self.V
        outs, states = [], []
        for s, n in enumerate(self.lengths):
            z = num(self.low[s]) @ num(self.a_up).T + num(self.bias)
            alpha = np.exp(-plain.softplus(-z) / self.tau).reshape(n, H, D)
            q, k = num(self.q[s]).reshape(n, H, D) * D ** -0.5, num(self.kk[s]).reshape(n, H, D)
            v = num(self.v[s]).reshape(n, H, V)
            o, S = zip(*(plain.gated_states(q[:, h], k[:, h], v[:, h], alpha[:, h], S=num(self.start[s][h])) for h in range(H)))
            o = plain.rms_unit(np.stack(o, axis=1), self.eps) * num(self.norm)
            outs.append(o.reshape(n, H * V) * plain.silu(num(self.g[s])))
            states.append(np.stack(S))
        return outs, states

    def run(self, cuts, slots, num_slots, step_kernel=True):
        k, H, D, V = self.k, self.H, self.D, self.V
        keys, inner, size = H * D, H * V, H * D * V
        state = torch.zeros(num_slots, -(-size // 4) * 4).cuda()
        spare = [i for i in range(num_slots) if i not in slots]
        for s, slot in enumerate(slots):
            state[slot, :size] = self.start[s].transpose(1, 2).reshape(-1).cuda()
        state[spare] = 7.0
        bias, norm, a_up = self.bias.cuda(), self.norm.cuda(), self.a_up.contiguous().cuda()
        status = torch.zeros(4, dtype=torch.int32).cuda()
        got = [np.zeros((n, inner)) for n in self.lengths]
        for spans, T, q_start, q_len, seq_slots in Steps(self.lengths, cuts, slots):
            wide = torch.cat([take(p, spans) for p in (self.q, self.kk, self.v)], dim=1)
            q, kk, v = wide[:, :keys], wide[:, keys : 2 * keys], wide[:, 2 * keys :]
            g, low = take(self.g, spans), take(self.low, spans)
            out = torch.zeros(T, inner, dtype=self.dt).cuda()
            if step_kernel and all(b - a == 1 for _, a, b in spans):
                assert k.gated_linear_step(q, kk, v, low, a_up, bias, D ** -0.5, self.tau, H, D, V, g, norm, self.eps, out,
                                           state, q_start, seq_slots, len(spans))
            else:
                z = (low.float() @ a_up.float().T).contiguous()
                records = torch.zeros(k.gated_linear_scratch(T, len(spans), H, D)).cuda()
                y = torch.zeros(T, inner).cuda()
                k.gated_linear_chunks(q, kk, v, z, bias, D ** -0.5, self.tau, H, D, V, records, state, y, q_start, q_len,
                                      seq_slots, len(spans), T, status)
                k.gated_group_norm(y, g, norm.repeat(H).contiguous(), self.eps, H, out, T, gate_after=k.GATE_SILU)
            give(got, spans, out)
        assert int(status[0]) == 0
        assert bool((state[spare] == 7.0).all()), "another slot's state has changed"
        return got, [num(state[slot, :size].view(H, V, D).transpose(1, 2)) for slot in slots]


LINEAR_SIZES = [(2, 16, 24, 8.0, 5), (3, 10, 7, 1.0, 8), (1, 6, 15, 3.5, 1), (4, 64, 128, 16.0, 16), (2, 96, 33, 16.0, 8), (2, 136, 12, 12.0, 20),
                (1, 200, 40, 4.0, 16), (1, 250, 9, 16.0, 3), (1, 264, 36, 20.0, 16), (1, 500, 20, 16.0, 8), (1, 128, 260, 16.0, 16)]


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("heads,dim,vdim,tau,rank", LINEAR_SIZES)
def test_gated_linear_attention_in_portions(dtype, heads, dim, vdim, tau, rank):
    """Portions of one token, of less than a chunk, of whole chunks and of many chunks and a bit beside each other, from
    states that are not zero; single tokens (their own kernel, with a head's columns over a cluster) among them."""
    lengths = [120, 66, 30]
    cuts = [[1, 1, 2, 33, 1, 64, 15, 1, 1, 1], [1, 2, 32, 1, 27, 1, 1, 1], [3, 1, 1, 1, 1, 20, 2, 1]]
    case = LinearCase(dtype, heads, dim, vdim, tau, rank, lengths, seed=heads + dim + vdim)
    gen = torch.Generator().manual_seed(4)
    case.start = [torch.randn(s.shape, generator=gen) for s in case.start]
    want, want_state = case.plain()
    got, state = case.run(cuts, slots=[3, 0, 5], num_slots=6)
    for s in range(3):
        close(torch.from_numpy(got[s]), want[s], dtype, f"sequence {s}", f32=4e-5)
        close(torch.from_numpy(state[s]), want_state[s], "float32", f"state of sequence {s}", f32=2e-5)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("memory,tau", [(8.0, 16.0), (-12.0, 1.0), (-60.0, 0.5)])
def test_gated_linear_decays_near_one_and_near_nothing(dtype, memory, tau):
    """Decays so close to 1 that the state remembers everything, and such that products of them underflow within a chunk."""
    lengths = [150, 70]
    case = LinearCase(dtype, 2, 40, 24, tau, 6, lengths, seed=9, memory=memory)
    case.start = [torch.ones(s.shape) for s in case.start]
    want, want_state = case.plain()
    for cuts in ([[150], [70]], [[40, 1, 109], [1] * 70], [[1] * 150, [64, 6]]):
        got, state = case.run(cuts, slots=[1, 0], num_slots=2)
        for s in range(2):
            close(torch.from_numpy(got[s]), want[s], dtype, f"sequence {s}", f32=1e-4)
            close(torch.from_numpy(state[s]), want_state[s], "float32", f"state of sequence {s}", f32=3e-5)


def test_gated_linear_step_of_many_sequences():
    """So many sequences that a head's columns stay in one CTA, and so few that a cluster shares them."""
    for count in (1, 3, 40):
        case = LinearCase("float32", 4, 48, 96, 16.0, 8, [1] * count, seed=count)
        gen = torch.Generator().manual_seed(4)
        case.start = [torch.randn(s.shape, generator=gen) for s in case.start]
        want, want_state = case.plain()
        got, state = case.run([[1]] * count, slots=list(range(count)), num_slots=count + 1)
        for s in range(count):
            close(torch.from_numpy(got[s]), want[s], "float32", f"sequence {s} of {count}", f32=2e-5)
            close(torch.from_numpy(state[s]), want_state[s], "float32", f"state {s} of {count}")


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("H,G,dim,vdim,D,rot", [(4, 2, 24, 20, 32, 16), (3, 1, 14, 30, 32, 10), (8, 2, 64, 64, 64, 64), (6, 6, 48, 48, 48, 48),
                                                (6, 0, 24, 24, 32, 24), (1, 1, 128, 96, 128, 32), (2, 1, 16, 16, 16, 0)])
def test_norm_over_the_projection_rotation_and_cache(dtype, H, G, dim, vdim, D, rot):
    """The mean square is over the real columns of all heads (the padding counts neither in the sum nor in the number);
    rows of no slot write nothing; without key heads only q changes."""
    from velox_b200.ops import kernels as k
    from velox_b200.parts.rope import RotaryHalf

    dt = DTYPES[dtype]
    gen = torch.Generator().manual_seed(H + D)
    T, pages, page, eps = 9, 6, 4, 1e-5
    raw = {n: torch.randn(T, heads * size, generator=gen).to(dt) for n, heads, size in (("q", H, dim), ("k", G, dim), ("v", G, vdim))}
    w = {n: 1.0 + 0.4 * torch.randn(heads * dim, generator=gen) for n, heads in (("q", H), ("k", G))}

    def padded(t, heads, size):
        out = t.new_zeros(*t.shape[:-1], heads, D)
        out[..., :size] = t.reshape(*t.shape[:-1], heads, size)
        return out.reshape(*t.shape[:-1], heads * D)

    rows = torch.cat([padded(raw["q"], H, dim), padded(raw["k"], G, dim), padded(raw["v"], G, vdim)], dim=1).cuda()
    positions = np.array([0, 1, 5, 17, 40, 63, 3, 2, 9])
    spec = dc.rot(rot, 30.0, (4.0, 1.0, 4.0, 64)) if rot else None
    cos = sin = None
    if rot:
        table = RotaryHalf({"head_dim": D, "rotary_dim": rot, "theta": 30.0, "max_position": 64, "scaling": spec["scaling"]}, {},
                           dt, torch.device("cuda"))
        cos, sin = table.cos, table.sin
    slots = np.array([4, 5, 6, 7, -1, 20, 21, 9, 10])
    k_cache, v_cache = [torch.full((pages, page, max(G, 1), D), 7.0, dtype=dt).cuda() for _ in range(2)]
    status = torch.zeros(4, dtype=torch.int32).cuda()
    k.norm_rope_store(rows, dev_int(positions), cos, sin, rot, padded(w["q"], H, dim).cuda(), padded(w["k"], G, dim).cuda() if G else None,
                      H * dim, G * dim, eps, dev_int(slots), k_cache, v_cache, T, H, G, D, status)
    assert int(status[0]) == 0

    def turned(name, heads):
        x = (plain.rms_unit(num(raw[name]), eps) * num(w[name])).reshape(T, heads, dim)
        if not rot:
            return x
        long = np.zeros((64, heads, dim))
        out = np.zeros_like(x)
        for t, pos in enumerate(positions):
            long[pos] = x[t]
            out[t] = plain.rotate_half(long, spec)[pos]
        return out

    close(rows[:, : H * D].view(T, H, D)[..., :dim], turned("q", H), dtype, "q")
    assert bool((rows[:, : H * D].view(T, H, D)[..., dim:] == 0).all())
    flat_k, flat_v = k_cache.view(-1, max(G, 1), D), v_cache.view(-1, max(G, 1), D)
    used = [s for s in slots if s >= 0]
    if G:
        live = slots >= 0
        close(flat_k[used][..., :dim], turned("k", G)[live], dtype, "k")
        close(flat_v[used][..., :vdim], num(raw["v"]).reshape(T, G, vdim)[live], dtype, "v", f32=0.0, bf16=0.0)
        assert bool((flat_k[used][..., dim:] == 0).all()) and bool((flat_v[used][..., vdim:] == 0).all())
    else:
        used = []
    rest = [s for s in range(pages * page) if s not in used]
    assert bool((flat_k[rest] == 7.0).all()) and bool((flat_v[rest] == 7.0).all())


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_pair_embedding_in_portions(dtype):
    """The row of (previous token, token): inside a portion, on its border, for a sequence's first token, in a slot that
    another sequence has left; products far above 32 bits; tokens that name a drawn one on the device."""
    from velox_b200.ops import kernels as k

    dt = DTYPES[dtype]
    gen = torch.Generator().manual_seed(3)
    vocab, width, buckets, mp, mc = 300, 72, 41, 1000003, 998244353
    table, pairs = torch.randn(vocab, width, generator=gen).to(dt), torch.randn(buckets + 1, width, generator=gen).to(dt)
    cfg = {"embedding": {"scale": 1.7, "bigram": {"buckets": buckets, "mul_prev": mp, "mul_cur": mc}}}
    W = {"embed": num(table), "bigram": num(pairs)}
    tokens = random_prompts(vocab, LENGTHS, seed=2)
    last = torch.full((6, 1), 123, dtype=torch.int32).cuda()
    fed = dev_int([tokens[0][5], 0, tokens[2][4]])
    status = torch.zeros(4, dtype=torch.int32).cuda()
    got = [np.zeros((n, width)) for n in LENGTHS]
    for spans, T, q_start, q_len, slots in Steps(LENGTHS, CUTS, [3, 0, 5]):
        flat = []
        for s, a, b in spans:
            ids = list(tokens[s][a:b])
            for i in range(a, b):
                if (s, i) == (0, 5):
                    ids[i - a] = -1   # row 0 of the tokens drawn before
                if (s, i) == (2, 4):
                    ids[i - a] = -3
            flat += ids
        positions = dev_int(np.concatenate([np.arange(a, b) for _, a, b in spans]))
        resid = torch.full((T + 2, width), 9.0).cuda()
        k.embed_pairs(table.cuda(), pairs.cuda(), mp, mc, 1.7, dev_int(flat), fed, positions, last, resid, q_start, q_len, slots,
                      len(spans), T, status)
        assert bool((resid[T:] == 9.0).all())
        give(got, spans, resid)
    assert int(status[0]) == 0
    for s in range(3):
        close(torch.from_numpy(got[s]), plain.embed(cfg, W, tokens[s]), "float32", f"sequence {s}", f32=2e-7)
    assert [int(last[i]) for i in (3, 0, 5)] == [t[-1] for t in tokens] and int(last[1]) == 123
    resid = torch.zeros(1, width).cuda()
    k.embed_pairs(table.cuda(), pairs.cuda(), mp, mc, 1.7, dev_int([vocab]), None, dev_int([0]), last, resid, dev_int([0]), dev_int([1]),
                  dev_int([0]), 1, 1, status)
    assert int(status[0]) == 1 and bool((resid == 0).all())


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("experts,top,width", [(6, 2, 64), (5, 5, 100), (9, 1, 40), (160, 8, 256), (33, 4, 72)])
def test_softmax_router(dtype, experts, top, width):
    """Biases that change the choice and count in the weights; large logits; from the input and from the logits."""
    from velox_b200.ops import kernels as k

    dt = DTYPES[dtype]
    gen = torch.Generator().manual_seed(experts + top)
    T = 70
    h = torch.randn(T, width, generator=gen).to(dt)
    w = (4.0 * torch.randn(experts, width, generator=gen) / width ** 0.5).to(dt)
    bias = 2.0 * torch.randn(experts, generator=gen) + 50.0
    margins = []
    picks = plain.route(num(h), {"router": num(w), "router.b": num(bias)}, "", {"top": top}, margins)
    logits = (h.double() @ w.double().T).float().cuda()
    for form in ("input", "logits"):
        chosen, weights = torch.full((T, top), -5, dtype=torch.int32).cuda(), torch.zeros(T, top).cuda()
        if form == "input":
            assert k.route_rows(h.cuda(), w.cuda(), bias.cuda(), 1, 1, top, 1.0, chosen, weights, T, router=k.ROUTER_SOFTMAX)
        else:
            k.choose_experts(logits, bias.cuda(), 1, 1, top, 1.0, chosen, weights, T, router=k.ROUTER_SOFTMAX)
        for t in range(T):
            if margins[t] > 1e-4:
                assert dict(zip(chosen[t].tolist(), weights[t].tolist())) == pytest.approx(dict(picks[t]), rel=1e-4), (form, t)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("width", [64, 100, 1536, 30])
def test_sums_join_behind_a_scaled_norm(dtype, width):
    """Float32 sums joined as ``x + m * rms_norm(sums) * w``, the copy of the rows in the compute dtype, and the sums
    handed back empty."""
    from velox_b200.ops import kernels as k
    from velox_b200.parts.norms import RMSNorm

    gen = torch.Generator().manual_seed(width)
    x, sums, w = torch.randn(7, width, generator=gen), torch.randn(7, width, generator=gen), torch.randn(width, generator=gen)
    norm = RMSNorm({"size": width, "eps": 1e-5, "weight_scale": 0.3}, {"weight": w.cuda()}, DTYPES[dtype], torch.device("cuda"))
    want = num(x) + 0.3 * plain.rms_unit(num(sums), 1e-5) * num(w)
    xd, sd = x.cuda(), sums.cuda()
    low = torch.zeros(7, width, dtype=DTYPES[dtype]).cuda()
    k.gated_norm_add(xd, xd, None, None, norm.weight, norm.eps, False, 5, lowp_out=low, sums=sd, compute_dtype=DTYPES[dtype])
    close(xd[:5], want[:5], "float32", "stream", f32=1e-6)
    close(low[:5], want[:5], dtype, "copy", f32=1e-6)
    assert bool((sd[:5] == 0).all()) and torch.equal(sd[5:].cpu(), sums[5:]) and torch.equal(xd[5:].cpu(), x[5:])


# ------------------------------------------------------------------------------ whole models
CASES = {
    "small": (dc.SMALL, 4, (5, 11, 17, 60, 100), 2.0),
    "odd": (dc.ODD, 16, (1, 9, 33, 70, 150), 1.5),
    "wide": (dc.WIDE, 64, (130, 3, 65, 300, 64), 2.0),
    "tall": (dc.TALL, 8, (2, 3, 1, 50, 24), 1.5),
}


def reference(cfg, tensors, tokens, collect=None):
    """(logits, which rows had no close call in any router)."""
    margins = []
    logits = plain.forward(cfg, dc.as_numpy(tensors), tokens, collect, margins)
    clear = np.ones(len(tokens), bool)
    for m in margins:
        clear &= m > CLEAR
    return logits, clear


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    out = {}
    for name, (cfg, page, lengths, sharp) in CASES.items():
        folder = str(tmp_path_factory.mktemp("demavik_" + name))
        tensors = dc.make_weights(cfg, seed=5 + len(name), sharp=sharp, rank=dc.RANKS[name])
        dc.write_folder(folder, cfg, tensors)
        prompts = random_prompts(cfg["vocab"], lengths, seed=31)
        want = [reference(cfg, tensors, p) for p in prompts]
        out[name] = (folder, cfg, page, prompts, want, tensors)
    return out


def make_replayer(folder, dtype, max_tokens, page, **kw):
    from velox_b200.engine.replay import TraceReplayer

    return TraceReplayer(folder, dtype, max_tokens, block_size=page, **kw)


def replay_one(replayer, name, tokens, cuts):
    rows, start = [], 0
    for step, n in enumerate(cuts):
        rec = {"step": step, "entries": [{"id": name, "tokens": tokens[start : start + n], "want": list(range(n))}],
               "end": [name] if start + n == len(tokens) else []}
        rows.append(replayer.run_step(rec))
        start += n
    assert start == len(tokens)
    return np.concatenate(rows, axis=0)


def changing_cuts(total):
    sizes = [7, 2, 16, 3, 2, 5, 33, 2, 9, 64, 4, 2, 21]
    cuts, left, i = [], total, 0
    while left > 0:
        n = min(sizes[i % len(sizes)], left)
        if left - n == 1:
            n = left
        cuts.append(n)
        left -= n
        i += 1
    return cuts


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("case", list(CASES))
def test_whole_then_decode_then_portions(models, case, dtype):
    folder, cfg, page, prompts, want, _ = models[case]
    longest = max(len(p) for p in prompts)
    replayer = make_replayer(folder, dtype, max_tokens=max(256, -(-longest // 64) * 64), page=page)
    for index, (tokens, (ref, clear)) in enumerate(zip(prompts, want)):
        L = len(tokens)
        whole = replay_one(replayer, f"w{index}", tokens, [L])
        check_logits(whole, ref, dtype, f"{case} request {index} whole", clear)
        tail = min(32, L - 1)
        if tail > 0:
            decoded = replay_one(replayer, f"d{index}", tokens, [L - tail] + [1] * tail)
            check_logits(decoded, ref, dtype, f"{case} request {index} last {tail} one by one", clear)
        if L > 2:
            portions = replay_one(replayer, f"p{index}", tokens, changing_cuts(L))
            check_logits(portions, ref, dtype, f"{case} request {index} in portions", clear)
        if L > 1:
            n = min(L, 24)
            each = replay_one(replayer, f"e{index}", tokens[:n], [1] * n)
            check_logits(each, ref[:n], dtype, f"{case} request {index} token by token from the start", clear[:n])
    replayer.cache.assert_consistent()
    assert replayer.cache.num_free_pages() == replayer.cache.num_total_pages
    assert replayer.cache.num_free_slots == replayer.max_live


@pytest.mark.parametrize("case", list(CASES))
def test_layer_streams(models, case):
    """The stream after every layer of the float32 path against the plain implementation's."""
    folder, cfg, page, prompts, _, tensors = models[case]
    tokens = prompts[3]
    streams = []
    reference(cfg, tensors, tokens, streams)
    replayer = make_replayer(folder, "float32", max_tokens=320, page=page, enable_graphs=False)
    seen = []
    for block in replayer.model.blocks:
        def wrapped(hidden, ctx, cache, inner=block.forward):
            inner(hidden, ctx, cache)
            assert hidden.delta is None
            seen.append(hidden.resid[: ctx.num_tokens].double().cpu())
        block.forward = wrapped
    replay_one(replayer, "s", tokens, [len(tokens)])
    assert len(seen) == len(streams) == len(cfg["layers"])
    for index, (got, want) in enumerate(zip(seen, streams)):
        close(got, want, "float32", f"stream after layer {index}", scale=8 * float(np.abs(want).max()))


def mixed_trace(prompts, rng, max_live=4):
    progress = [0] * len(prompts)
    waiting = list(range(len(prompts)))
    live, steps = [], []
    step = 0
    while waiting or live:
        while waiting and len(live) < max_live:
            live.append(waiting.pop(0))
        entries, ends = [], []
        single = rng.random() < 0.3          # a step of single tokens only, not all of them wanted
        for r in list(live):
            left = len(prompts[r]) - progress[r]
            if rng.random() < 0.2 and len(live) > 1:
                continue
            decoding = single or left <= 12 or rng.random() < 0.3
            n = 1 if decoding else min(left, int(rng.choice([2, 3, 5, 8, 13, 30])))
            if left - n == 0:
                ends.append(r)
            entries.append((r, progress[r], n))
            progress[r] += n
        if not entries:
            continue
        steps.append((step, entries, ends))
        for r in ends:
            live.remove(r)
        step += 1
    return steps


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("case", list(CASES))
def test_mixed_batches_with_pages_and_slots_used_again(models, case, dtype):
    """Every request twice, up to four live at a time in a pool that holds no more: a request's
    logits equal those of the request alone whatever shares its steps, and a slot's previous token, convolution
    inputs and recurrent states and a page's keys of an earlier request do not leak into a later one.
    Every third step wants only its last place."""
    folder, cfg, page, prompts, want, _ = models[case]
    order = list(range(len(prompts))) * 2
    seqs = [prompts[i] for i in order]
    steps = mixed_trace(seqs, np.random.default_rng(9))
    need = sum(sorted((-(-len(p) // 64) * 64 for p in prompts), reverse=True)[:4])
    replayer = make_replayer(folder, dtype, max_tokens=need, page=page, max_live=4)
    got = [np.zeros((len(p), cfg["vocab"]), np.float32) for p in seqs]
    seen = [np.zeros(len(p), bool) for p in seqs]
    slots_used = []
    for step, entries, ends in steps:
        wants = [list(range(n)) if step % 3 else ([n - 1] if step % 2 else []) for _, _, n in entries]
        rec = {"step": step, "end": [f"r{r}" for r in ends],
               "entries": [{"id": f"r{r}", "tokens": seqs[r][s : s + n], "want": w} for (r, s, n), w in zip(entries, wants)]}
        out = replayer.run_step(rec)
        row = 0
        for (r, s, n), w in zip(entries, wants):
            for place in w:
                got[r][s + place] = out[row]
                seen[r][s + place] = True
                row += 1
        slots_used.extend(seq.slot for seq in replayer.live.values())
        replayer.cache.assert_consistent()
    for r, ref_index in enumerate(order):
        ref, clear = want[ref_index]
        if seen[r].any():
            check_logits(got[r][seen[r]], ref[seen[r]], dtype, f"{case} mixed request {r}", clear[seen[r]])
    assert replayer.cache.num_free_pages() == replayer.cache.num_total_pages
    assert set(slots_used) <= set(range(4))


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("case,page", [("small", 4), ("wide", 16)])
def test_long_decode(models, case, page, dtype):
    """390 tokens one by one: the recurrent states run through 420 updates, pages are taken one after the other."""
    folder, cfg, _, _, _, tensors = models[case]
    tokens = random_prompts(cfg["vocab"], [420], seed=4)[0]
    ref, clear = reference(cfg, tensors, tokens)
    replayer = make_replayer(folder, dtype, max_tokens=448, page=page)
    rows = replay_one(replayer, "long", tokens, [30] + [1] * 390)
    check_logits(rows, ref, dtype, "long decode", clear)
    replayer.cache.assert_consistent()


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("case", ["wide", "small"])
def test_long_prompt_whole_and_in_large_portions(models, case, dtype):
    """Steps of more than 512 tokens (the scan's chunks side by side), of more than the projections' small-step limit (the
    library's products, experts through its grouped product) and shorter ones of the same prompt."""
    folder, cfg, page, _, _, tensors = models[case]
    tokens = random_prompts(cfg["vocab"], [1100], seed=14)[0]
    ref, clear = reference(cfg, tensors, tokens)
    replayer = make_replayer(folder, dtype, max_tokens=1152, page=page)
    check_logits(replay_one(replayer, "whole", tokens, [1100]), ref, dtype, "1,100 tokens whole", clear)
    check_logits(replay_one(replayer, "parts", tokens, [600, 298, 2, 199, 1]), ref, dtype, "1,100 tokens in portions", clear)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("case", ["small", "odd", "tall"])
def test_first_tokens(models, case, dtype):
    """The first tokens have no token before them, fewer inputs than the convolutions have taps, and zero states."""
    folder, cfg, page, prompts, want, _ = models[case]
    ref, clear = want[3]
    replayer = make_replayer(folder, dtype, max_tokens=64, page=page)
    for name, cuts in (("one by one", [1, 1, 2, 2, 1]), ("in portions", [2, 5]), ("as long as the taps", [3, 1, 3]),
                       ("single tokens", [1] * 7), ("whole", [7])):
        rows = replay_one(replayer, name, prompts[3][:7], cuts)
        check_logits(rows, ref[:7], dtype, "first tokens " + name, clear[:7])


MARKER, ASKER, WIDTH, VOCAB = 7, 11, 64, 90


def model_of(layers, bigram=None, seed=2):
    cfg = dc.config(WIDTH, VOCAB, layers, eps=1e-6, mult=1.0, scale=2.0, bigram=bigram)
    return cfg, {k: v.float() for k, v in dc.make_weights(cfg, seed=seed, rank=8).items()}


def written(tmp_path, cfg, tensors, name="model"):
    tensors = {k: v.to(torch.bfloat16) for k, v in tensors.items()}
    folder = str(tmp_path / name)
    dc.write_folder(folder, cfg, tensors)
    return folder, tensors


def stream_row(tensors, token):
    return 2.0 * tensors["embed"][token]


def pointed_prompt(length, needle_at, ask_at, seed):
    tokens = [t if t not in (MARKER, ASKER) else 20 for t in random_prompts(VOCAB, [length], seed=seed)[0]]
    tokens[needle_at], tokens[ask_at] = MARKER, ASKER
    without = list(tokens)
    without[needle_at] = 21
    return tokens, without


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("ask_at,needle_at", [(319, 318), (319, 0), (319, 63), (319, 64), (319, 65), (300, 127), (320, 128), (321, 191),
                                              (64, 0), (65, 1), (2, 1)])
def test_a_key_that_takes_nearly_all_weight(tmp_path, dtype, shared, ask_at, needle_at):
    """Attention: one key scores far above the others for one query: the first key, keys at page and tile borders, the
    key just before; the query decoded alone, at the end and inside of portions, and whole.  ``shared``: the
    keys are another layer's, whose own queries see nothing of the kind."""
    rotation = dc.rot(8, 50.0, (4.0, 1.0, 4.0, 64))
    layers = [dc.layer("attention", dc.attn(2, 2, 16, 16, 0.25, rotation), None)]
    if shared:
        layers.append(dc.layer("attention", dc.attn(4, 2, 16, 16, 0.25, rotation, kv_from=0), None))
    cfg, tensors = model_of(layers)
    if shared:
        tensors["l0.norm1"].zero_()   # the first layer only provides the keys: the stream passes it unchanged
    asking = "l1.mix." if shared else "l0.mix."
    # one dimension behind the rotated ones lines the two tokens up; the norms over the projections keep its share
    for name, p, token in (("q", asking, ASKER), ("k", "l0.mix.", MARKER)):
        v = stream_row(tensors, token)
        tensors[p + name][12] = 25.0 * v / float(v @ v)
        tensors[p + name + ".b"][12] = 0.0
        tensors[p + name + ".norm"][12] = 2.5
    folder, tensors = written(tmp_path, cfg, tensors)
    length = 330 if ask_at > 100 else 80
    tokens, without = pointed_prompt(length, needle_at, ask_at, seed=needle_at)
    ref, _ = reference(cfg, tensors, tokens)
    other, _ = reference(cfg, tensors, without)
    assert float(np.abs(other[ask_at] - ref[ask_at]).max()) > 0.3, "the key does not matter enough for this test"
    lo, hi = max(ask_at - 3, 0), ask_at + 4
    for page in (64, 16):
        replayer = make_replayer(folder, dtype, max_tokens=384, page=page)
        for cuts in ([ask_at, 1, length - ask_at - 1], [ask_at - 1, 2, length - ask_at - 1], [length],
                     [ask_at // 2, ask_at - ask_at // 2 + 5, length - ask_at - 5]):
            rows = replay_one(replayer, str(cuts), tokens, cuts)
            check_logits(rows[lo:hi], ref[lo:hi], dtype, f"key at {needle_at}, pages of {page}, {cuts}")


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("kind", ["gla", "mamba1"])
def test_a_write_is_recalled_hundreds_of_tokens_later(tmp_path, kind, dtype):
    """A state that hardly decays and into which hardly any token but one writes: what that one wrote 600 tokens ago
    is read by a query made to ask for it, across chunks, portions, pages and decoded tokens."""
    mixer = dc.gla(2, 16, 24, 16.0) if kind == "gla" else dc.mamba(48, 6, 4, 2)
    cfg, tensors = model_of([dc.layer(kind, mixer, None)])
    # one coordinate of the stream is the marker's alone, one the asker's
    tensors["embed"][:, :2] = 0.0
    tensors["embed"][MARKER, 0] = tensors["embed"][ASKER, 1] = 2.0
    gen = torch.Generator().manual_seed(5)
    p = "l0.mix."
    if kind == "gla":
        tensors[p + "a2"].zero_()
        tensors[p + "a2.b"].fill_(14.0)
        key = torch.randn(32, generator=gen)
        tensors[p + "k"], tensors[p + "q"] = 0.01 * tensors[p + "k"], 0.05 * tensors[p + "q"]
        tensors[p + "k"][:, 0], tensors[p + "q"][:, 1] = key, key
    else:
        # the first two channels read those coordinates; the marker's step size is large, the others' next to nothing
        tensors[p + "conv"][:, 0] = 0.0
        tensors[p + "conv"][:, 1] = 1.0
        tensors[p + "conv.b"].zero_()
        tensors[p + "A_log"].fill_(-6.0)
        tensors[p + "D"].zero_()
        tensors[p + "in"][:2] = 0.0
        tensors[p + "in"][0, 0] = tensors[p + "in"][1, 1] = 2.0
        tensors[p + "x"].zero_()
        tensors[p + "x"][0, 0] = 1.5
        tensors[p + "x"][4:10, 0] = 0.2 * torch.randn(6, generator=gen)
        tensors[p + "x"][10:16, 1] = 0.2 * torch.randn(6, generator=gen)
        tensors[p + "dt"].zero_()
        tensors[p + "dt"][:, 0] = 1.0
        tensors[p + "dt.b"].fill_(-9.0)
    folder, tensors = written(tmp_path, cfg, tensors)
    length, needle_at, ask_at = 700, 40, 655
    tokens, without = pointed_prompt(length, needle_at, ask_at, seed=3)
    ref, _ = reference(cfg, tensors, tokens)
    other, _ = reference(cfg, tensors, without)
    assert float(np.abs(other[ask_at] - ref[ask_at]).max()) > 0.3, "the write does not matter enough for this test"
    lo, hi = ask_at - 3, ask_at + 4
    replayer = make_replayer(folder, dtype, max_tokens=704, page=16)
    for cuts in ([length], [ask_at, 1, length - ask_at - 1], [20] + [1] * 60 + [570] + [1] * 50, [30, 2, 2, 2, 2, 2, 2, 600, 10, 2, 2, 44]):
        rows = replay_one(replayer, str(len(cuts)) + str(cuts[0]), tokens, cuts)
        # (in bfloat16 only the asker's own row: the others' read-outs are next to nothing before they are normed)
        rows_at = slice(ask_at, ask_at + 1) if dtype == "bfloat16" else slice(lo, hi)
        check_logits(rows[rows_at], ref[rows_at], dtype, f"{kind} memory, {len(cuts)} steps")


EDGE_CUTS = lambda at, back: ([40], [at, 1, 39 - at], [at - back, back + 3, 37 - at], [at - 1, 2, 39 - at], [at - 2] + [1] * 6 + [36 - at], [1] * 40)


@pytest.mark.parametrize("dtype", list(DTYPES))
@pytest.mark.parametrize("conv", [4, 2, 1])
def test_the_edges_of_the_convolution(tmp_path, conv, dtype):
    """A state that forgets everything at once: a token's output depends on the tokens its taps reach and on no
    other.  The token taps - 1 back matters, the one taps back does not; the edge lies inside a portion, on
    its border and among decoded tokens."""
    cfg, tensors = model_of([dc.layer("mamba1", dc.mamba(48, 4, 4, conv), None)])
    tensors["l0.mix.dt.b"].fill_(60.0)
    tensors["l0.mix.A_log"].fill_(2.0)
    tensors["l0.mix.x"][8:12] = tensors["l0.mix.x"][4:8]   # C = B: the state's share cannot nearly cancel the input's
    tensors["l0.mix.D"].fill_(1.0)
    tensors["l0.mix.conv"][:, 0] = 1.5 * torch.sign(tensors["l0.mix.conv"][:, 0])
    folder, tensors = written(tmp_path, cfg, tensors)
    tokens = random_prompts(VOCAB, [40], seed=8)[0]
    at = 25
    ref, _ = reference(cfg, tensors, tokens)
    for back, matters in ((conv - 1, True), (conv, False)):
        changed = list(tokens)
        changed[at - back] = (changed[at - back] + 31) % VOCAB
        other, _ = reference(cfg, tensors, changed)
        moved = float(np.abs(other[at] - ref[at]).max())
        assert (moved > 0.1) if matters else (moved < 1e-6), (back, moved)
        replayer = make_replayer(folder, dtype, max_tokens=64, page=4)
        for cuts in EDGE_CUTS(at, conv):
            rows = replay_one(replayer, str(cuts), changed, cuts)
            check_logits(rows[at - 2 : at + 3], other[at - 2 : at + 3], dtype, f"{back} back, {cuts}")


@pytest.mark.parametrize("dtype", list(DTYPES))
def test_the_edge_of_the_pair_embedding(tmp_path, dtype):
    """The token right before matters, the one before it does not (in a layer that forgets at once); on a portion's border
    and among decoded tokens the token before comes from the request's state."""
    cfg, tensors = model_of([dc.layer("mamba1", dc.mamba(48, 4, 4, 1), None)], bigram=(61, 12, 5))
    tensors["l0.mix.dt.b"].fill_(60.0)
    tensors["l0.mix.A_log"].fill_(2.0)
    tensors["l0.mix.x"][8:12] = tensors["l0.mix.x"][4:8]   # C = B: the state's share cannot nearly cancel the input's
    tensors["l0.mix.D"].fill_(1.0)
    folder, tensors = written(tmp_path, cfg, tensors)
    tokens = random_prompts(VOCAB, [40], seed=18)[0]
    at = 25
    ref, _ = reference(cfg, tensors, tokens)
    for back, matters in ((1, True), (2, False)):
        changed = list(tokens)
        changed[at - back] = (changed[at - back] + 31) % VOCAB
        other, _ = reference(cfg, tensors, changed)
        moved = float(np.abs(other[at] - ref[at]).max())
        assert (moved > 0.1) if matters else (moved < 1e-6), (back, moved)
        replayer = make_replayer(folder, dtype, max_tokens=64, page=4)
        for cuts in EDGE_CUTS(at, 2):
            rows = replay_one(replayer, str(cuts), changed, cuts)
            check_logits(rows[at - 2 : at + 3], other[at - 2 : at + 3], dtype, f"{back} back, {cuts}")


def test_command_lines_take_the_design(tmp_path, capsys):
    import json

    from velox_b200.cli import benchmark, roofline

    common = ["--model-size", "tiny-d", "--num-requests", "5", "--max-tokens", "10", "--max-model-len", "128",
              "--max-num-seqs", "4", "--max-num-batched-tokens", "64", "--max-prefill-chunk-size", "16",
              "--block-size", "8", "--workload", "short", "--seed", "3"]
    assert benchmark.main(common + ["--temperature", "0"]) == 0
    assert "decode throughput" in capsys.readouterr().out
    assert benchmark.main(common + ["--temperature", "0.7", "--top-k", "10", "--no-pipeline"]) == 0
    capsys.readouterr()
    table = tmp_path / "roofline.json"
    assert roofline.main(["--model-size", "tiny-d", "--batch", "2", "--context", "40", "--layers", "4,8", "--steps", "4",
                          "--warmup", "1", "--block-size", "8", "--output-json", str(table)]) == 0
    rows = json.loads(table.read_text())
    assert rows[0]["us_per_layer"] > 0 and rows[0]["size"] == "tiny-d"


@pytest.mark.parametrize("case", ["small", "odd", "tall"])
def test_greedy_generation_through_the_engine(models, case):
    """The engine's own entry point: its scheduler cuts prompts into portions of 8 beside decoding
    requests, two requests at a time, greedy sampling; the tokens drawn are fed on the device, the pair embedding's
    previous token with them."""
    from velox_b200.engine.engine import LLM
    from velox_b200.sampling.params import SamplingParams

    folder, cfg, page, prompts, _, tensors = models[case]
    asks = [prompts[1], prompts[2], prompts[0], prompts[3]]
    for dtype in ("float32", "bfloat16"):
        llm = LLM(folder, dtype=dtype, max_model_len=96, max_num_seqs=2, max_num_batched_tokens=24,
                  max_prefill_chunk_size=8, block_size=page, num_gpu_blocks=max(8, 320 // page))
        outputs = llm.generate(asks, SamplingParams(temperature=0.0, max_tokens=9, ignore_eos=True))
        for prompt, output in zip(asks, outputs):
            assert len(output) == 9
            rows, clear = reference(cfg, tensors, prompt + output[:-1])
            rows, clear = rows[len(prompt) - 1 :], clear[len(prompt) - 1 :]
            if dtype == "float32":
                assert output == rows.argmax(-1).tolist()
            else:
                for row, token, sure in zip(rows, output, clear):
                    if sure:
                        assert row[token] >= row.max() - 6e-2 * np.abs(row).max()
