"""The Zinurax kernels one by one against plain expressions, with inputs made so that one wrong key, one lost state or one
misplaced row dominates the result."""
import math

import pytest
import torch

from oracle import zinurax_oracle as Z

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module", autouse=True)
def _lib_built():
    from megatron_mixtera_b200 import build

    build.build_torch_ops()


def rand(*shape, seed=0, dtype=torch.float32):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)).to(dtype)


# ---------------------------------------------------------------------------------------------------------------------
# linears and norms
# ---------------------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,N,K", [(1, 8, 8), (5, 77, 30), (70, 130, 72), (300, 256, 200), (33, 264, 1024)])
@pytest.mark.parametrize("act", [None, "relu2"])
def test_linear(dtype, M, N, K, act):
    from megatron_mixtera_b200 import ops

    x, w = rand(M, K, seed=1, dtype=dtype), rand(N, K, seed=2, dtype=dtype) / math.sqrt(K)
    w = w.to(dtype)
    want = x.double() @ w.double().T
    want = torch.relu(want).square() if act else want
    got = ops.linear(x.to(DEV), w.to(DEV), act=act).cpu().double()
    tol = 1e-5 if dtype == torch.float32 else 8e-3
    assert (got - want).abs().max() <= tol * want.abs().max()
    if dtype == torch.bfloat16 and act is None:  # fp32 partial sums for a consumer that reduces
        p = ops.linear_partials(x.to(DEV), w.to(DEV))
        parts = p.buf[: 4 * p.num_splits * M * N].view(torch.float32).view(p.num_splits, M, N).sum(0).cpu().double()
        assert (parts - want).abs().max() <= 1e-5 * want.abs().max()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("M,heads,N,K,gap", [(3, 5, 40, 24, 16), (70, 4, 200, 72, 8), (9, 3, 11, 10, 6), (130, 2, 256, 128, 64)])
def test_batched_linear(dtype, M, heads, N, K, gap):
    """One product per head out of and into wider rows; what lies between the heads' columns must not leak in."""
    from megatron_mixtera_b200 import ops

    x = rand(M, heads * (K + gap) + 8, seed=3, dtype=dtype)
    w = (rand(heads * N, K, seed=4) / math.sqrt(K)).to(dtype)
    out = torch.full((M, heads * (N + 5)), 7.0, dtype=dtype, device=DEV)
    ops.linear(x.to(DEV), w.to(DEV), out=out, batch=heads, x_batch=K + gap, y_batch=N + 5, K=K)
    for h in range(heads):
        want = x[:, h * (K + gap): h * (K + gap) + K].double() @ w[h * N: (h + 1) * N].double().T
        got = out[:, h * (N + 5): h * (N + 5) + N].cpu().double()
        assert (got - want).abs().max() <= (1e-5 if dtype == torch.float32 else 8e-3) * want.abs().max()
        assert bool((out[:, h * (N + 5) + N: (h + 1) * (N + 5)] == 7.0).all())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width", [32, 100, 1000, 2048, 8192, 9001])
def test_out_norm(dtype, width):
    """All three sources; a large common offset, which a one-pass variance would lose."""
    from megatron_mixtera_b200 import ops

    eps, rows = 1e-5, 7
    gamma = (1 + 0.2 * rand(width, seed=5)).to(dtype)
    table = (50.0 + rand(19, width, seed=6)).to(dtype)
    ids = torch.tensor([3, 0, 18, 3, 7, 1, 2])
    want = Z.layer_norm(table[ids].double(), gamma.double(), eps)
    hidden = torch.empty(rows, width, device=DEV)
    y = ops.out_norm(table.to(DEV), gamma.to(DEV), eps=eps, hidden=hidden, ids=ids.to(DEV))
    assert (hidden.cpu() - want).abs().max() < 2e-4
    assert y.dtype == dtype and (y.float().cpu() - want).abs().max() < (2e-4 if dtype == torch.float32 else 0.04)

    parts = rand(3, rows, width, seed=7) + 20.0
    p = ops.GemmPartials(parts.to(DEV).view(-1).view(torch.uint8), 3, (rows, width))
    before = hidden.clone()
    ops.out_norm(p, gamma.to(DEV), eps=eps, hidden=hidden, accumulate=True)
    want = before.cpu().double() + Z.layer_norm(parts.double().sum(0), gamma.double(), eps)
    assert (hidden.cpu() - want).abs().max() < 2e-4

    pick = torch.tensor([6, 2, 2])
    y = ops.out_norm(hidden, gamma.to(DEV), eps=eps, row_index=pick.to(DEV))
    want = Z.layer_norm(hidden.cpu().double()[pick], gamma.double(), eps)
    assert (y.float().cpu() - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.04)


def test_argmax_of_fp32_logits():
    from megatron_mixtera_b200 import ops

    x = rand(6, 5001, seed=8)
    x[2, 17] = x[2, 4000] = 9.0  # equal maxima: the smaller index
    x[3] = x[3, 0] + torch.arange(5001) * 1e-7  # differences bf16 cannot see
    assert ops.argmax(x.to(DEV)).cpu().tolist() == [int(r.argmax()) if i != 2 else 17 for i, r in enumerate(x)]


# ---------------------------------------------------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------------------------------------------------
class Paged:
    """A pool with scattered chunks, and the arguments of the latent kernels over it."""

    def __init__(self, lengths, kv_rank, rot, heads, window, dtype, chunk=64, seed=0, dim=8):
        from megatron_mixtera_b200.transformer.hybrid_config import LatentAttentionConfig, RotaryConfig

        self.m = LatentAttentionConfig(heads=heads, dim=dim, rot_dim=rot, vdim=8, kv_rank=kv_rank, scale=0.3,
                                       rot=RotaryConfig(base=10000.0, dims=rot // 2 * 2), window=window)
        self.lengths, self.dtype, self.chunk = lengths, dtype, chunk
        self.rows = [rand(n, kv_rank + rot, seed=seed + 100 + i, dtype=dtype) for i, n in enumerate(lengths)]
        need = [-(-n // chunk) for n in lengths]
        perm = torch.randperm(sum(need) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
        self.table = torch.zeros(len(lengths), max(need), dtype=torch.int32)
        self.num_chunks = sum(need) + 3
        for i, n in enumerate(need):
            self.table[i, :n] = torch.tensor([perm.pop() for _ in range(n)], dtype=torch.int32)

    def pool(self):
        m = self.m
        pool = torch.full((self.num_chunks, self.chunk, m.row_width), float("nan"), dtype=self.dtype)  # unused places poison
        for i, rows in enumerate(self.rows):
            for j in range(rows.shape[0]):
                pool[self.table[i, j // self.chunk], j % self.chunk] = self.padded(rows[j])
        return pool.to(DEV)

    def padded(self, row):
        m = self.m
        out = torch.zeros(*row.shape[:-1], m.row_width, dtype=self.dtype)
        out[..., : m.kv_rank] = row[..., : m.kv_rank]
        out[..., m.kv_pad: m.kv_pad + m.rot_dim] = row[..., m.kv_rank:]
        return out

    def want(self, q, row, pos):
        """q [heads, kv_rank + rot] at position pos of request row -> [heads, kv_rank]."""
        lo = 0 if self.m.window is None else max(0, pos - self.m.window + 1)
        keys = self.rows[row][lo: pos + 1].double()
        p = torch.softmax(q.double() @ keys.T * self.m.scale, dim=-1)
        return p @ keys[:, : self.m.kv_rank]

    def args(self, T, q_full, pool, gates, out):
        from megatron_mixtera_b200 import _lib, ops

        m, a = self.m, _lib.LatentArgs()
        self.d_table = self.table.to(DEV)
        a.proj, a.proj_ld, a.gate_offset, a.dkv_offset = gates.data_ptr(), gates.stride(0), 0, -1
        a.block_table, a.max_chunks_per_row = self.d_table.data_ptr(), self.table.shape[1]
        a.pool, a.num_chunks, a.chunk_size = pool.data_ptr(), self.num_chunks, self.chunk
        a.q_full, a.out, a.num_tokens = q_full.data_ptr(), out.data_ptr(), T
        a.heads, a.dim, a.rot_dim, a.rot_dims, a.kv_rank, a.kv_pad, a.row_width = (
            m.heads, m.dim, m.rot_dim, m.rot.dims, m.kv_rank, m.kv_pad, m.row_width)
        a.window, a.scale, a.eps, a.dtype, a.num_splits = m.window or 0, m.scale, 1e-5, ops.dtype_code(self.dtype), 1
        return a


def stand_out(pg, q, row, pos, key, head, strength=12.0):
    """Turn one head's query towards one key, so that the key outweighs all others together."""
    k = pg.rows[row][key].float()
    q[head] = (k * (strength / pg.m.scale / float(k @ k))).to(q.dtype)


SHAPES = [  # kv_rank, rot, heads, window
    (96, 16, 5, 33), (512, 64, 16, 150), (512, 64, 40, 150), (512, 64, 72, 70), (128, 32, 32, None), (256, 64, 1, 64),
    (72, 24, 20, 7), (36, 6, 3, 50), (40, 8, 17, 1), (200, 56, 12, 300), (640, 64, 4, 90)]
LIMIT = {torch.float32: 2e-5, torch.bfloat16: 1e-2}


def compare(got, want, dtype):
    assert torch.isfinite(got.float()).all()
    err = (got.float().cpu().double() - want).abs().max() / want.abs().max()
    assert err < LIMIT[dtype], float(err)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", SHAPES)
def test_latent_decode_attention(dtype, shape):
    """Rows of many lengths in one launch, for several split counts; per row one head looks at the key just inside the
    window (or the first), one at the key just outside, one at a key at a chunk's border."""
    from megatron_mixtera_b200 import ops

    kv_rank, rot, heads, window = shape
    lengths = [1, 2, 63, 64, 65, 128, 129, 333]
    pg = Paged(lengths, kv_rank, rot, heads, window, dtype)
    T = len(lengths) + 1  # one padding row
    q = rand(T, heads, kv_rank + rot, seed=9, dtype=dtype) * 0.1
    for i, n in enumerate(lengths):
        pos = n - 1
        for h, key in enumerate([max(0, n - (window or n)), n - (window or n) - 1, 64, 63, 0]):
            if h < heads and 0 <= key <= pos:
                stand_out(pg, q[i], i, pos, key, h)
    pg.table = torch.cat([pg.table, torch.zeros(1, pg.table.shape[1], dtype=torch.int32)])
    gates = rand(T, heads, seed=10, dtype=dtype)
    pool, qf = pg.pool(), pg.padded(q).to(DEV)
    kv_len = torch.tensor(lengths + [0], dtype=torch.int32, device=DEV)
    want = torch.stack([pg.want(q[i], i, n - 1) for i, n in enumerate(lengths)]) * torch.sigmoid(gates[:-1].double())[:, :, None]
    g = gates.to(DEV)
    for splits in (1, 2, 5):
        out = torch.empty(T, heads, kv_rank, dtype=dtype, device=DEV)
        a = pg.args(T, qf, pool, g, out)
        a.kv_seq_lengths, a.num_splits = kv_len.data_ptr(), splits
        ops.latent_attention(a, pool)
        compare(out[:-1], want, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("shape", SHAPES)
def test_latent_prompt_attention(dtype, shape):
    """Portions that start anywhere: at the first token, inside a chunk, one token before an edge."""
    from megatron_mixtera_b200 import ops

    kv_rank, rot, heads, window = shape
    lengths, begin = [40, 130, 200, 65], [0, 63, 198, 64]
    pg = Paged(lengths, kv_rank, rot, heads, window, dtype, seed=1)
    where = [(r, p) for r in range(4) for p in range(begin[r], lengths[r])]
    T = len(where)
    q = rand(T, heads, kv_rank + rot, seed=11, dtype=dtype) * 0.1
    for t, (r, p) in enumerate(where):
        for h, key in enumerate([max(0, p + 1 - (window or p + 1)), p - (window or p), p, 0]):
            if h < heads and 0 <= key <= p:
                stand_out(pg, q[t], r, p, key, h)
    units, t0 = [], 0
    for r in range(4):
        for k in range(0, lengths[r] - begin[r], 16):
            units.append((r, t0 + k, min(16, lengths[r] - begin[r] - k), 0))
        t0 += lengths[r] - begin[r]
    units += [(0, 0, 0, 0)] * 2  # empty entries of a fixed-size list
    d_units = torch.tensor(units, dtype=torch.int32, device=DEV)
    gates = rand(T, heads, seed=12, dtype=dtype)
    pos = torch.tensor([p for _, p in where], device=DEV)
    pool, qf, g = pg.pool(), pg.padded(q).to(DEV), gates.to(DEV)
    out = torch.empty(T, heads, kv_rank, dtype=dtype, device=DEV)
    a = pg.args(T, qf, pool, g, out)
    a.units, a.num_units, a.unit_tokens, a.token_to_pos = d_units.data_ptr(), len(units), 16, pos.data_ptr()
    ops.latent_attention(a, pool)
    want = torch.stack([pg.want(q[t], r, p) for t, (r, p) in enumerate(where)]) * torch.sigmoid(gates.double())[:, :, None]
    compare(out, want, dtype)


@pytest.mark.parametrize("heads,dim,rot,vdim,window", [(5, 24, 16, 40, 33), (3, 128, 64, 128, None), (20, 8, 24, 16, 7), (2, 64, 32, 64, 1),
                                                       (1, 112, 8, 8, 150), (4, 16, 64, 72, 64)])
def test_latent_prompt_attention_on_expanded_keys(heads, dim, rot, vdim, window):
    """Gathered rows and the attention on spelled-out keys and values: rows that start and that continue, a row without
    tokens, heads that look at the key just inside the window, the one just outside, the token itself and the first."""
    from megatron_mixtera_b200 import ops

    dtype, kv_rank, chunk = torch.bfloat16, 48, 64
    lengths, begin = [40, 130, 64, 200], [0, 63, 64, 137]
    pg = Paged(lengths, kv_rank, rot, heads, window, dtype, chunk=chunk, seed=2, dim=dim)
    m = pg.m
    first = [0 if window is None else max(0, b - window + 1) for b in begin]
    first[2] = 64  # no tokens, no keys
    cu_t, cu_k = [0], [0]
    for r in range(4):
        cu_t.append(cu_t[-1] + lengths[r] - begin[r])
        cu_k.append(cu_k[-1] + lengths[r] - first[r])
    T, E = cu_t[-1], cu_k[-1]
    keys, vals = rand(E, heads, dim, seed=50, dtype=dtype) * 0.3, rand(E, heads, vdim, seed=51, dtype=dtype)
    q = rand(T, heads, dim + rot, seed=52, dtype=dtype) * 0.1
    gates = rand(T, heads, seed=53, dtype=dtype)
    want = torch.empty(T, heads, vdim, dtype=torch.float64)
    for r in range(4):
        for t in range(cu_t[r], cu_t[r + 1]):
            pos = begin[r] + t - cu_t[r]
            lo = 0 if window is None else max(0, pos - window + 1)
            rows = torch.arange(cu_k[r] + lo - first[r], cu_k[r] + pos - first[r] + 1)
            full = torch.cat([keys[rows], pg.rows[r][lo: pos + 1, None, kv_rank:].expand(-1, heads, -1)], -1)
            for h, key in enumerate([max(lo, pos + 1 - (window or pos + 1)), lo - 1, pos, 0]):
                if h < heads and lo <= key <= pos:
                    k = full[key - lo, h].float()
                    q[t, h] = (k * (12.0 / m.scale / float(k @ k))).to(dtype)
            p = torch.softmax(torch.einsum("hd,khd->hk", q[t].double(), full.double()) * m.scale, -1)
            want[t] = torch.einsum("hk,khv->hv", p, vals[rows].double()) * torch.sigmoid(gates[t].double())[:, None]
    proj = torch.zeros(T, heads * (dim + rot) + -(-heads // 8) * 8, dtype=dtype)
    proj[:, : heads * (dim + rot)] = q.reshape(T, -1)
    proj[:, heads * (dim + rot): heads * (dim + rot) + heads] = gates
    q_rot = torch.zeros(T, heads, m.row_width - m.kv_pad, dtype=dtype)
    q_rot[..., :rot] = q[..., dim:]
    kv = torch.cat([keys.reshape(E, -1), vals.reshape(E, -1)], 1).contiguous()
    pool = pg.pool()
    d = [t.to(DEV) for t in (proj, q_rot, kv, torch.tensor(cu_t, dtype=torch.int32), torch.tensor(cu_k, dtype=torch.int32),
                             torch.tensor(first, dtype=torch.int32))]
    key_rows = torch.empty(E, m.row_width, dtype=dtype, device=DEV)
    out = torch.empty(T, heads, vdim, dtype=dtype, device=DEV)
    a = pg.args(T, d[1], pool, d[0], out)
    a.gate_offset, a.q_stride, a.q_rot_at, a.vdim = heads * (dim + rot), m.row_width - m.kv_pad, 0, vdim
    a.cu_tokens, a.cu_keys, a.key_start, a.key_rows, a.key_values = (d[3].data_ptr(), d[4].data_ptr(), d[5].data_ptr(),
                                                                     key_rows.data_ptr(), d[2].data_ptr())
    a.num_rows, a.num_keys, a.max_row_tokens = 4, E, max(lengths[r] - begin[r] for r in range(4))
    assert ops.latent_prompt_supported(dim, rot, vdim, heads)
    ops.latent_gather(a, pool)
    plain = torch.cat([pg.padded(pg.rows[r][first[r]: lengths[r]]) for r in range(4)])
    assert torch.equal(key_rows.cpu(), plain)
    ops.latent_prompt_attention(a, pool)
    compare(out, want, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kv_rank,rot,dims,heads,dim", [(96, 16, 16, 5, 24), (36, 6, 6, 3, 12), (72, 24, 10, 2, 8), (512, 64, 64, 16, 128)])
def test_latent_append(dtype, kv_rank, rot, dims, heads, dim):
    """Normed latent and rotated key part in their place in the pool, nothing else touched; rotated queries; far positions."""
    from megatron_mixtera_b200 import _lib, ops
    from megatron_mixtera_b200.transformer.hybrid_config import LatentAttentionConfig, RotaryConfig, YarnScaling
    from megatron_mixtera_b200.transformer.rotary import rotary_tables

    rc = RotaryConfig(base=5000.0, dims=dims, scaling=YarnScaling(4.0, 96, 8.0, 1.0))
    plain = {"base": 5000.0, "dims": dims, "scaling": {"factor": 4.0, "original": 96, "fast": 8.0, "slow": 1.0}}
    m = LatentAttentionConfig(heads=heads, dim=dim, rot_dim=rot, vdim=8, kv_rank=kv_rank, scale=1.0, rot=rc)
    pos = torch.tensor([0, 1, 77, 1500, 2047])
    T, eps = len(pos), 1e-5
    q_w = heads * (dim + rot)
    proj = rand(T, q_w + kv_rank + rot + heads, seed=13, dtype=dtype)
    norm = (1 + 0.2 * rand(kv_rank, seed=14)).to(dtype)
    chunk, local = torch.tensor([2, 0, 1, 2, 1]), torch.tensor([0, 63, 5, 1, 6])
    pool = torch.full((3, 64, m.row_width), 3.0, dtype=dtype, device=DEV)
    qf = torch.full((T, heads, m.row_width), 3.0, dtype=dtype, device=DEV)
    cos, sin = rotary_tables(rc, 2048, DEV)
    d = [t.to(DEV) for t in (proj, norm, pos, chunk, local)]
    a = _lib.LatentArgs()
    a.proj, a.proj_ld, a.dkv_offset, a.gate_offset = d[0].data_ptr(), proj.shape[1], q_w, -1
    a.norm_weight, a.rope_cos, a.rope_sin, a.max_positions = d[1].data_ptr(), cos.data_ptr(), sin.data_ptr(), 2048
    a.token_to_pos, a.token_to_chunk_idx, a.token_to_local_pos = (t.data_ptr() for t in d[2:])
    a.pool, a.num_chunks, a.chunk_size, a.q_full, a.num_tokens = pool.data_ptr(), 3, 64, qf.data_ptr(), T
    a.heads, a.dim, a.rot_dim, a.rot_dims, a.kv_rank, a.kv_pad, a.row_width = heads, dim, rot, dims, kv_rank, m.kv_pad, m.row_width
    a.eps, a.dtype, a.q_stride, a.q_rot_at = eps, ops.dtype_code(dtype), m.row_width, m.kv_pad
    ops.latent_append(a, pool)
    tol = 2e-5 if dtype == torch.float32 else 2e-2
    lat = proj[:, q_w: q_w + kv_rank + rot].double()
    rows = torch.zeros(T, m.row_width, dtype=torch.float64)
    rows[:, :kv_rank] = Z.rms_norm(lat[:, :kv_rank], norm.double(), eps)
    rows[:, m.kv_pad: m.kv_pad + rot] = Z.rotate(lat[:, kv_rank:], pos, plain)
    for t in range(T):
        assert (pool[chunk[t], local[t]].cpu().double() - rows[t]).abs().max() < tol * rows.abs().max()
    untouched = torch.ones(3, 64, dtype=torch.bool)
    untouched[chunk, local] = False
    assert bool((pool.cpu()[untouched] == 3.0).all())
    want_q = Z.rotate(proj[:, :q_w].double().view(T, heads, dim + rot)[..., dim:].contiguous(), pos, plain)
    assert (qf[..., m.kv_pad: m.kv_pad + rot].cpu().double() - want_q).abs().max() < tol * want_q.abs().max()
    assert bool((qf[..., m.kv_pad + rot:] == 0).all()) and bool((qf[..., kv_rank: m.kv_pad] == 0).all())
    assert bool((qf[..., :kv_rank] == 3.0).all())  # the absorbed part belongs to the batched GEMM


# ---------------------------------------------------------------------------------------------------------------------
# generalized delta rule
# ---------------------------------------------------------------------------------------------------------------------
class DeltaCase:
    def __init__(self, heads, dim, rank, T, dtype, seed=0):
        n = heads * dim
        self.heads, self.dim, self.rank, self.n, self.T, self.dtype = heads, dim, rank, n, T, dtype
        self.proj = rand(T, 5 * n + rank, seed=seed + 1, dtype=dtype)
        self.w2 = (rand(n, rank, seed=seed + 2) / math.sqrt(rank)).to(dtype)
        self.w0 = (-2.0 + 2.0 * rand(n, seed=seed + 3)).to(dtype)
        self.ab = rand(n, seed=seed + 4, dtype=dtype)
        self.norm = (1 + 0.2 * rand(n, seed=seed + 5)).to(dtype)
        self.dev = [t.to(DEV) for t in (self.proj, self.w2, self.w0, self.ab, self.norm)]

    def inputs(self, lo, hi):
        """(r, k, v, decay, removal, unit key) of tokens [lo, hi) from the plain expressions."""
        p, n, shape = self.proj[lo:hi].double(), self.n, (hi - lo, self.heads, self.dim)
        r, k, v, a = (p[:, i * n: (i + 1) * n].reshape(shape) for i in (0, 1, 2, 4))
        z = torch.tanh(p[:, 5 * n:]) @ self.w2.double().T + self.w0.double()
        decay = torch.exp(-math.exp(-0.5) * torch.sigmoid(z)).view(shape)
        a = torch.sigmoid(a.reshape(hi - lo, n) + self.ab.double()).view(shape)
        return r, k, v, decay, a, k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)

    def finish(self, o, lo, hi, eps):
        y = Z.rms_norm(o, None, eps).reshape(hi - lo, self.n) * self.norm.double()
        return y * torch.sigmoid(self.proj[lo:hi, 3 * self.n: 4 * self.n].double())

    def args(self, state, rd, wr, out, eps=1e-5):
        from megatron_mixtera_b200 import _lib, ops

        a = _lib.DeltaArgs()
        a.proj, a.proj_ld = self.dev[0].data_ptr(), self.proj.shape[1]
        a.w2, a.decay_bias, a.removal_bias, a.norm_weight = (t.data_ptr() for t in self.dev[1:])
        a.state, a.state_slots, a.state_in, a.state_out = state.data_ptr(), state.shape[0], rd.data_ptr(), wr.data_ptr()
        a.out, a.rank, a.heads, a.dim = out.data_ptr(), self.rank, self.heads, self.dim
        a.off_r, a.off_k, a.off_v, a.off_g, a.off_a, a.off_w1 = (i * self.n for i in range(6))
        a.num_tokens = a.num_rows = self.T
        a.dtype, a.decay_scale, a.unit_eps, a.eps = ops.dtype_code(self.dtype), math.exp(-0.5), 1e-6, eps
        return a


DELTA_SHAPES = [(3, 48, 24), (2, 64, 16), (1, 128, 8), (3, 20, 5), (1, 256, 16), (4, 32, 64), (2, 100, 12), (1, 8, 3), (5, 2, 1)]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,rank", DELTA_SHAPES)
def test_delta_decode(dtype, heads, dim, rank):
    """One token per row from an existing state, from none, and a padding row; read and written buffers differ, so the same
    step run again gives the same bits."""
    from megatron_mixtera_b200 import ops

    c = DeltaCase(heads, dim, rank, 4, dtype)
    state = rand(9, heads, dim, dim, seed=20)
    old = state.clone()
    rd, wr = torch.tensor([2, -1, 5, -1], dtype=torch.int32), torch.tensor([3, 0, 8, -1], dtype=torch.int32)
    d_state, d_rd, d_wr = state.to(DEV), rd.to(DEV), wr.to(DEV)
    runs = []
    for _ in range(2):
        out = torch.full((4, c.n), 9.0, dtype=dtype, device=DEV)
        ops.delta_decode(c.args(d_state, d_rd, d_wr, out), d_state)
        runs.append((out.cpu(), d_state.cpu()))
    assert torch.equal(runs[0][0], runs[1][0]) and torch.equal(runs[0][1], runs[1][1])
    out, new = runs[0]
    for row in range(3):
        S0 = old[rd[row]].double().transpose(1, 2) if rd[row] >= 0 else None  # stored [value channel][key channel]
        o, S = Z.delta_scan(*c.inputs(row, row + 1), state=S0)
        got = new[wr[row]].double().transpose(1, 2)
        assert (got - S).abs().max() < 2e-5 * S.abs().max()
        want = c.finish(o, row, row + 1, 1e-5)
        assert (out[row].double() - want).abs().max() < (1e-4 if dtype == torch.float32 else 1e-2) * want.abs().max()
    keep = [i for i in range(9) if i not in wr.tolist()]
    assert torch.equal(new[keep], old[keep])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("heads,dim,rank", DELTA_SHAPES)
def test_delta_scan(dtype, heads, dim, rank):
    """Rows of 1, 2, 16, 17 and 40 tokens and an empty one in one launch, some continuing from a state."""
    from megatron_mixtera_b200 import ops

    lens = [1, 17, 0, 40, 2, 16]
    T, pad = sum(lens), 4
    c = DeltaCase(heads, dim, rank, T + pad, dtype, seed=30)
    cu = torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
    state = rand(12, heads, dim, dim, seed=31)
    rd = torch.tensor([0, -1, -1, 4, 6, -1], dtype=torch.int32)
    wr = torch.tensor([1, 3, -1, 5, 7, 9], dtype=torch.int32)
    d_state, d_rd, d_wr = state.to(DEV), rd.to(DEV), wr.to(DEV)
    out = torch.empty(T + pad, c.n, dtype=dtype, device=DEV)
    o_f32 = torch.zeros(T + pad, c.n, device=DEV)
    lora = torch.empty(T + pad, rank, dtype=dtype, device=DEV)
    a = c.args(d_state, d_rd, d_wr, out)
    a.num_rows, a.cu_tokens, a.o_f32, a.lora = len(lens), cu.data_ptr(), o_f32.data_ptr(), lora.data_ptr()
    ops.delta_lora(a, d_state)
    z = ops.linear(lora, c.dev[1])
    a.z = z.data_ptr()
    ops.delta_scan(a, d_state)
    ops.delta_finish(a, d_state)
    new, at = d_state.cpu(), 0
    tol = 1e-4 if dtype == torch.float32 else 2e-2  # bf16: tanh and the decay's projection are rounded
    for row, n in enumerate(lens):
        if n == 0:
            continue
        S0 = state[rd[row]].double().transpose(1, 2) if rd[row] >= 0 else None
        o, S = Z.delta_scan(*c.inputs(at, at + n), state=S0)
        assert (new[wr[row]].double().transpose(1, 2) - S).abs().max() < tol * S.abs().max()
        want = c.finish(o, at, at + n, 1e-5)
        assert (out[at: at + n].cpu().double() - want).abs().max() < tol * want.abs().max()
        at += n


def test_delta_state_survives_long_rows():
    """A value written at the first token with decay close to one is still there 600 tokens later, and only there."""
    from megatron_mixtera_b200 import ops

    heads, dim, rank, T = 2, 64, 8, 600
    c = DeltaCase(heads, dim, rank, T, torch.float32, seed=40)
    n = c.n
    c.w0 = torch.full((n,), -12.0)           # decay = exp(-0.6 * sigmoid(-12)): forgets 0.2 % in 600 tokens
    c.ab = torch.full((n,), -30.0)           # nothing is removed
    c.proj[1:, 2 * n: 3 * n] = 0.0           # only the first token carries a value
    c.proj[-1, :n] = c.proj[0, n: 2 * n]     # the last token asks for the first one's key
    c.dev = [t.to(DEV) for t in (c.proj, c.w2, c.w0, c.ab, c.norm)]
    state = torch.zeros(2, heads, dim, dim, device=DEV)
    rd, wr = torch.tensor([-1], dtype=torch.int32, device=DEV), torch.tensor([1], dtype=torch.int32, device=DEV)
    cu = torch.tensor([0, T], dtype=torch.int32, device=DEV)
    out, o_f32 = torch.empty(T, n, device=DEV), torch.empty(T, n, device=DEV)
    z = ops.linear(torch.tanh(c.dev[0][:, 5 * n:]).contiguous(), c.dev[1])
    a = c.args(state, rd, wr, out)
    a.num_rows, a.cu_tokens, a.o_f32, a.z = 1, cu.data_ptr(), o_f32.data_ptr(), z.data_ptr()
    ops.delta_scan(a, state)
    k0 = c.proj[0, n: 2 * n].view(heads, dim)
    v0 = c.proj[0, 2 * n: 3 * n].view(heads, dim)
    want = (v0 * (k0 * k0).sum(-1, keepdim=True)).view(-1)
    got = o_f32[-1].cpu()
    assert (got - want).abs().max() < 5e-3 * want.abs().max()
