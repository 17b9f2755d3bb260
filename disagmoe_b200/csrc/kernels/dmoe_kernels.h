// C ABI of libdmoe_kernels.so: hand-written sm_100a kernels of the serving engine.
// Every function takes raw device pointers and a CUDA stream handle and returns 0 on success, a positive
// cudaError_t, or a negative argument error. Nothing here allocates device memory unless it says so.
#pragma once
#include <stdint.h>

#ifdef __cplusplus
extern "C" {

// Router of dmoe_sum_norm (weight [E, W] in the activations' dtype): softmax scores or, sigmoid = 1, sigmoid scores with a
// correction (NULL: none) that enters the choice, not the weight, within the best `keep` of `groups` runs of E / groups experts.
typedef struct DmoeRouter {
  const void* weight;
  const float* correction;  // [E]
  int* ids;                 // [rows, K]
  float* wts;               // [rows, K]: scores, with renorm divided by their sum, times wscale
  int* counts;              // [E], may be NULL
  int E, K, renorm, sigmoid, groups, keep;
  float wscale;
} DmoeRouter;
// Token shift: n_mix outputs h + (before - h) mu per row, `before` = the row before in the sequence, kept per slot in `last`.
// singles: int4 {row, 1, slot, position}; NULL: one-token segment i is row i, as in DmoeRecur.
typedef struct DmoeShift {
  const float* mu;          // [n_mix, W]
  float* last;              // [n_slots, W]
  const void* singles;
  const int* positions;
  const int* rows;
  const long long* kv_slots;
  long long mix_stride;     // elements from one output to the next
  int n_mix, n_slots, n_single;
} DmoeShift;
// Causal convolution over time per channel: sum_j w[j] x_(t - taps + 1 + j) + out_bias of the inputs x + in_bias, with `residual` plus
// the input itself. The last inputs (without their bias) of a sequence sit in its slot's ring by position modulo taps. blocks: the
// output columns are cut into equal blocks, stored one after the other in rows of `padded` numbers. Singles as in DmoeShift.
typedef struct DmoeConv {
  const float* w;           // [taps, C]
  const float* in_bias;     // [C], may be NULL
  const float* out_bias;
  void* ring;               // [n_slots, taps, C]
  const void* singles;
  const int* positions;
  const int* rows;
  const long long* kv_slots;
  int n_single, n_slots, taps, residual, blocks, padded;
} DmoeConv;
// Further steps of dmoe_sum_norm (all optional): a bias of the norm [W]; what is added to the residual is multiplied by
// sigmoid(gate_z[row] + gate_bias); `side`: two rows per row instead of y, added up as side_scale * their RMS norms times side_w [2, W];
// conv (all rows one-token segments): the second output, one matrix of n rows after h, is the convolution of h.
typedef struct DmoeSumExtra {
  const float* bias;
  const void* gate_z;
  const float* gate_bias;
  const void* side;
  const float* side_w;
  const DmoeConv* conv;
  long long ld_gate, ld_side, side_stride;
  float side_scale;
} DmoeSumExtra;
// Options of the attention kernels: head outputs times sigmoid(gate[row, head]) (NULL: none), scores times the query temperature
// 1 + temp_coef ln(floor((p + 1) / temp_every) + 1) of the query's position p (temp_every 0: none).
typedef struct DmoeAttnExtra {
  const void* gate;
  long long ld_gate;
  float temp_coef;
  int temp_every;
} DmoeAttnExtra;
// Real-gated diagonal recurrence (diag_recurrent.cu): u [blocks, block_rows, padded], gate logits [blocks, block_rows, 2, padded] with
// biases [blocks, 2, padded], y and out [rows, width]; state [n_slots, width]; segment tables as in DmoeRecur.
typedef struct DmoeUnit {
  const void* u;
  const float* gates;
  const float* gate_bias;
  const float* decay;       // [width] log decay of an open gate
  const void* y;
  const float* y_bias;
  float* state;
  void* out;
  const void* singles;
  const int* positions;
  const int* rows;
  const long long* kv_slots;
  const void* multi;
  long long ldy, ldo, block_rows;
  int n_single, n_multi, n_slots, width, blocks, padded;
} DmoeUnit;
#endif

// ---- GEMM (gemm.cu) -------------------------------------------------------------------------------
// Y[t, f] = sum_k X[t, k] * W[g][f, k] for t in group g. bf16 inputs, fp32 accumulation.
enum { DMOE_EPI_PLAIN = 0, DMOE_EPI_SWIGLU = 1, DMOE_EPI_COMBINE = 2 };

typedef struct DmoeGemm {
  const void* W;      // [G, rows, K] bf16; rows = F (plain / combine) or 2F (SwiGLU: gate rows then up rows)
  const void* X;      // [T, K] bf16, row stride ldx (0 = K)
  void* Y;            // [T, F] bf16 (or fp32 when y_f32), row stride ldy; unused for combine
  const void* R;      // optional residual [T, F] bf16, row stride ldr (plain epilogue only)
  const int* offs;    // [G+1] device token offsets of the groups, or NULL for one dense group
  const void* recs;   // combine: [T] int4 {dst_rank, dst_row (<0 = drop), weight as fp32 bits, 0}
  const void* bases;  // combine: device array of destination base pointers (bf16 rows of stride ldy), one per rank
  void* ws;           // split-K workspace (fp32), ws_bytes >= dmoe_gemm_workspace_bytes(...)
  int* counters;      // split-K tile counters, zero-initialised once; the kernel leaves them zero
  int* status;        // optional device status word (0 = ok)
  // --- multi-GPU fusion (all optional, zero / NULL when unused) ---
  const int* seg_cnt;   // [S, G] rows that source s delivered for group g; region s = rows [s*seg_cap, (s+1)*seg_cap)
  const int* wait_flags;  // [n_wait] arrival flags written by peers; the kernel waits for *wait_epoch + 1
  int* wait_epoch;
  const void* signal_ptrs;  // device array of n_signal flag-array pointers (peer memory); slot signal_slot is written
  int* signal_epoch;
  int* done_ticket;     // one zero-initialised int of scratch (required with wait_flags or signal_ptrs)
  long long ldx, ldy, ldr, ws_bytes;
  int S, seg_cap, n_wait, n_signal, signal_slot;
  int group_regions;    // 1: group g owns rows [g*seg_cap, (g+1)*seg_cap) and seg_cnt[g] is its row count (S unused)
  int clear_n;          // the last CTA zeroes clear_ptr[0..clear_n) before it signals (the dispatch cursors)
  int* clear_ptr;
  int fanout;           // combine: every row is stored to the `fanout` consecutive ranks of the sender's TP group (0/1 = one)
  int G, T, F, K;
  int epi;            // DMOE_EPI_*
  int bn;             // token tile: 32/64/128/256, 0 = pick from T/G
  int splitk;         // >= 1; > 1 only for dense plain / combine GEMMs
  int y_f32;
  // --- tensor-parallel attention fusion (plain epilogue with 16-byte aligned Y; all optional) ---
  // all-gather prologue: rows [s * shard_rows, (s + 1) * shard_rows) of X are pushed by peer s, which then sets
  // wait_flags[s]; a token tile is fetched as soon as the shards it covers have landed (n_wait = number of shards)
  int shard_rows;
  // reduce-scatter epilogue: row t is stored to row rs_slot * rs_cap + t % rs_rows of buffer rs_bases[t / rs_rows]
  // (device array of peer pointers, row stride ldy) instead of Y
  const void* rs_bases;
  int rs_rows, rs_slot, rs_cap;
  // QKV epilogue: neox RoPE on the n_q + n_kv leading heads of head size hd (64 / 128) from rope_table
  // ([rope_max_pos][hd / 2] float2 = (cos, sin), see dmoe_rope_table), K / V rows appended to the paged caches
  // ([blocks, block_size, n_kv, hd]) at slots[t] (< 0: skip); only the q columns are written to Y. F = (n_q + 2 n_kv) hd.
  const void* rope_table;
  const int* positions;
  const long long* slots;
  void* kcache;
  void* vcache;
  int n_q, n_kv, hd, rope_max_pos;
  // --- work distribution ---
  // streamk != 0 (with splitk <= 1, ws and counters given): the K-block iterations of all tiles are dealt out in one
  // equal contiguous share per CTA instead of whole tiles, so no SM idles in a last partial wave; tiles that straddle
  // a share boundary are reduced through ws (2 slots of 128 x bn fp32 per accumulator and CTA). n_counters: ints
  // available at `counters` (0 = 4096); one per tile is needed.
  int streamk, n_counters;
  // pair != 0: clusters of two CTAs compute tiles of 256 weight rows x bn tokens with tcgen05.mma.cta_group::2 (each
  // CTA stages its 128 weight rows and half of the token tile). bn = 128 or 256 (SwiGLU too), whole tiles only.
  int pair;
  // combine epilogue: != 0 states that every destination base in `bases` is 16-byte aligned (with F and ldy multiples
  // of 8 the rows then move as 16-byte segments); 0 keeps 2-byte stores
  int combine_vec;
  // != 0: W is stored tile by tile, [group][128-row tile][K / 64][128][64] (see ops/gemm.py: block_weight), so that
  // every 16 KB box the kernel fetches is one contiguous run of HBM; needs F % 128 == 0 and K % 64 == 0
  int w_blocked;
  // gate activation of the SwiGLU epilogue: 0 silu, 1 gelu (tanh form), 3 clamped: min(g, act_limit) sigmoid(1.702 g)
  // (clamp(u, act_limit) + 1); plain epilogue: 2 = tanh of the output, 4 = silu of its first act_cols columns. SwiGLU with
  // recs: gate and up of row t are multiplied by the weight of record t first.
  int act;
  // profiling aid, normally null: 16 x uint64 of device memory that CTA 0 fills with %globaltimer stamps (entry, set-up
  // done, first TMA issued, first stage landed, last MMA committed, accumulator seen by the epilogue, epilogue done,
  // tear-down reached, then five points inside the first epilogue chunk and three inside the producer's start)
  void* trace;
  float act_limit;
  int act_cols;
  int unit_weights;   // combine: the records' weights are left out
} DmoeGemm;

int dmoe_gemm(const DmoeGemm* desc, void* stream);
int dmoe_gemm_pick_bn(int tokens_per_group_hint, int epi);
long long dmoe_gemm_workspace_bytes(int T, int F, int bn, int splitk);

// ---- row kernels (elementwise.cu) -------------------------------------------------------------------
// resid_out = resid_in + sum of n_add partial rows; y = rmsnorm(resid_out) * w. resid_in / resid_out / y may be NULL.
int dmoe_add_rmsnorm(const void* resid_in, const void* add, int n_add, long long add_row_stride,
                     long long add_part_stride, const void* w, float eps, void* resid_out, void* y, int T, int H,
                     long long ld_in, long long ld_out, long long ld_y, void* stream);
// neox RoPE on the q and k heads of qkv rows [q | k | v] in place, then K/V append at slots[t] (slot < 0: no append).
int dmoe_rope_kv_append(void* qkv, long long ld, const int* positions, const long long* slots, void* kcache,
                        void* vcache, int T, int n_q, int n_kv, int hd, float theta, void* stream);
// (cos, sin) of pos * theta^(-2 d / hd) for pos < max_pos, d < hd / 2: the table the QKV epilogue rotates with.
int dmoe_rope_table(void* table, int max_pos, int hd, float theta, void* stream);
int dmoe_embed(const int* ids, const void* table, void* out, int T, int H, int vocab, long long ld_out, void* stream);
int dmoe_argmax(const void* logits, int is_f32, long long ld, int T, int V, int* ids, void* stream);
int dmoe_permute_rows(const void* src, long long ld_src, void* dst, long long ld_dst, const int* map, int n, int H,
                      int repeat, int gather, void* stream);
int dmoe_gather_ptrs(const void* ptrs, void* dst, long long ld_dst, int n, int H, void* stream);
// Debug kernel of the launch / overlap tests: out[i] = in[i] + 1 (fp32).
int dmoe_add_one(const float* in, float* out, long long n, void* stream);

// ---- attention (attention.cu) -----------------------------------------------------------------------
long long dmoe_paged_attention_workspace_floats(int T, int n_q, int hd, int splits);
int dmoe_paged_attention(const void* q, long long ld_q, const void* kcache, const void* vcache,
                         const int* block_tables, int max_blocks, const int* bt_row, const int* ctx_len, int block_size,
                         int T, int n_q, int n_kv, int hd, float scale, int splits, void* out, long long ld_out,
                         float* workspace, void* stream);

// With a sliding window (a query sees the last `window` tokens, itself included; 0 = all), a score soft cap
// (cap * tanh(score / cap); 0 = none) and a sink (exp(sink[head]) enters the softmax denominator; NULL = none); value heads
// of size vd. (hd, vd) = (64, 32), (64, 64), (64, 128), (128, 64), (128, 128), up to 64 query heads per kv head.
int dmoe_paged_attention_ext(const void* q, long long ld_q, const void* kcache, const void* vcache, const int* block_tables,
                             int max_blocks, const int* bt_row, const int* ctx_len, int block_size, int T, int n_q, int n_kv,
                             int hd, int vd, float scale, int window, int chunk, float softcap, const float* sink, int splits, void* out,
                             long long ld_out, float* workspace, const DmoeAttnExtra* extra, void* stream);
int dmoe_prefill_attention_ext(const void* q, long long ld_q, const void* kcache, const void* vcache,
                               const int* block_tables, int max_blocks, const void* tiles, int n_tiles, int block_size,
                               int n_q, int n_kv, int hd, int vd, float scale, int window, int chunk, float softcap, const float* sink,
                               void* out, long long ld_out, const DmoeAttnExtra* extra, void* stream);
// Any key / value size and query group, bf16 or fp32 cache, fp32 arithmetic on the CUDA cores. Query i of head h starts at
// q + i * q_row + h * q_head (output likewise) and has the context of batch row rows[i] (NULL: i); the heads of a cached token
// are contiguous, tokens k_tok / v_tok elements apart.
int dmoe_any_attention(int is_f32, const void* q, long long q_head, long long q_row, const void* kcache, long long k_tok,
                       const void* vcache, long long v_tok, const int* block_tables, int max_blocks, const int* bt_row,
                       const int* rows, const int* ctx_len, int block_size, int T, int n_q, int n_kv, int dk, int dv,
                       float scale, int window, int chunk, float softcap, const float* sink, void* out, long long o_head, long long o_row,
                       const DmoeAttnExtra* extra, void* stream);

// ---- latent attention (latent_attention.cu): the cache has one row [latent rankp | rotated key part rotp] per token,
// `row` elements apart ------
// Projection rows y = [heads x (q dimp | rotp) | latent rankp | key part rotp] (every part padded to a multiple of 8): RMS norm
// of the latent, rotation of the key part, both to cache rows at slots (< 0: skip); rotation of the queries in place, and for
// rows with loose[t] = i >= 0 (NULL: i = t) to xq [heads, n_loose, dimp] and columns rankp.. of qa [heads, n_loose, row].
// gate (NULL: none; row stride ld): sigmoid(gate[t, h]) becomes the weight of record h * n_loose + i of recs (see DmoeGemm).
int dmoe_latent_prep(int is_f32, void* y, long long ld, const int* positions, const long long* slots, void* cache, int T,
                     int heads, int dim, int rot_dim, int rank, int row, int rot, int interleaved, const void* table, int max_pos,
                     const float* norm_w, float eps, const int* loose, int n_loose, void* xq, void* qa, const void* gate, void* recs, void* stream);
// Queries qa [heads, n, row] over cache rows (keys: the first kd columns, values: the first rankp), out [heads, n, rankp];
// rankp <= 512, kd <= 640, row an odd multiple of 8, block_size a multiple of 16. workspace: heads * n * splits * (rankp + 1) floats where splits > 1. status (may be NULL): non-zero
// after a bounded wait gave up.
int dmoe_latent_attention(const void* qa, const void* cache, const int* block_tables, int max_blocks, const int* bt_row,
                          const int* rows, const int* ctx_len, int block_size, int n, int heads, int rankp, int kd, int row,
                          float scale, int window, const float* sink, int splits, void* out, float* workspace, int* status, void* stream);
// out[i] = cache row of position keys[i].y of block-table row keys[i].x
int dmoe_latent_gather(const void* cache, const int* block_tables, int max_blocks, const void* keys, int n, int block_size,
                       int row, void* out, void* stream);
// Prompt tiles over expanded keys and values: tile i's key at position p is row base[i] + p of kv [heads x (dimp | vdimp)] and
// of lat (columns rankp ..: its rotated part). gate (NULL: none): head h's output is scaled by sigmoid(gate[row, h]).
int dmoe_latent_prefill(const void* q, long long ld_q, const void* kv, long long ld_kv, const void* lat, long long ld_lat,
                        const void* tiles, const int* base, int n_tiles, int heads, int dimp, int rotp, int rankp, int vdimp,
                        float scale, int window, const float* sink, const void* gate, long long ld_gate, void* out, long long ld_out,
                        void* stream);

// Tiled causal attention for prompt tokens: CTA column i handles tiles[i] = int4 {first row in q / out, tokens
// (<= dmoe_prefill_tile_tokens), block-table row, position of the first token}; the tokens of a tile are consecutive
// rows at consecutive positions of one sequence, whose K / V (own tokens included) are already in the paged cache.
int dmoe_prefill_tile_tokens(int n_q, int n_kv);
int dmoe_prefill_attention(const void* q, long long ld_q, const void* kcache, const void* vcache,
                           const int* block_tables, int max_blocks, const void* tiles, int n_tiles, int block_size,
                           int n_q, int n_kv, int hd, float scale, void* out, long long ld_out, void* stream);

// ---- fp32-residual decoders (layer_ops.cu); is_f32: fp32 activations instead of bf16 -----------------------
// out[t] = table[ids[t]] * scale (+ pos_table[positions[t]] where given, n_pos rows) (fp32)
int dmoe_embed_f32(const int* ids, const void* table, int is_f32, float scale, float* out, int T, int W, int vocab,
                   const int* positions, const void* pos_table, int n_pos, void* stream);
// x = resid[r] + norm(y[r]) * post (y may be NULL: x = resid[r]); resid[r] = x unless a row table picks r = rows[i];
// h[i] = norm(x) * pre * out_scale (h may be NULL); norm(v) = v / sqrt(mean(v^2) + eps). resid fp32 [.., W].
int dmoe_resid_norm(int is_f32, float* resid, const void* y, long long ld_y, const float* post, const float* pre,
                    float out_scale, float eps, const int* rows, void* h, long long ld_h, int n, int W, void* stream);
// float2 table [max_pos][half] = (cos, sin)(pos * freq[i]) * mscale, freq in double on the device
int dmoe_rope_freq_table(void* table, int max_pos, int half, const double* freq, float mscale, void* stream);
// Per-head RMS norm of q and k (qw, kw; NULL: none), rotation of pairs (i, i + rot / 2), i < rot / 2, or (2i, 2i + 1) where
// interleaved; q in place, k / v into the paged caches, v as (1 - v_lambda) v + v_lambda v_first where that is given
// (row stride ld_first, head stride first_head). tied: rows [q | k], the values are the first dv dimensions of the k heads before
// their rotation. v_norm > 0: every value head is divided by its root mean square over v_norm dimensions (the rest is zeros).
int dmoe_qk_norm_rope(int is_f32, void* qkv, long long ld, const int* positions, const long long* slots, void* kcache,
                      void* vcache, int T, int n_q, int n_kv, int dk, int dv, int rot, int interleaved, const void* table,
                      int max_pos, const float* qw, const float* kw, float eps, const void* v_first, long long ld_first,
                      int first_head, float v_lambda, int tied, int v_norm, void* stream);
// x = resid[r] + mult (y[r] + sum of n_parts rows of parts) (both may be NULL); resid[r] = x unless a row table picks
// r = rows[i]; h[i] = norm(x) * w, RMS norm or with `centred` layer norm, as fp32 where h_f32. router: the K best experts of
// every h and, where counts is given, the histogram of the chosen ones; E <= 256, K <= 32. shift (all rows one-token segments):
// h gets the n_mix mixed rows instead.
int dmoe_sum_norm(int is_f32, float* resid, const void* y, long long ld_y, const void* parts, int n_parts,
                  long long part_row, long long part_stride, float mult, const float* w, int centred, float eps, const int* rows,
                  void* h, int h_f32, long long ld_h, int n, int W, const DmoeRouter* router, const DmoeShift* shift, const DmoeSumExtra* extra,
                  void* stream);
// The token shift of a batch with longer segments (tables as in DmoeRecur: segs of the longer ones, their chunks): fp32 rows h ->
// n_mix outputs; the slots keep the last row of every segment.
int dmoe_token_shift(int is_f32, const float* h, const DmoeShift* s, const void* multi, int n_multi, const void* chunks, int n_chunks,
                     void* out, long long ld, int W, void* stream);
int dmoe_seq_conv(int is_f32, const void* x, long long ldx, const DmoeConv* a, const void* multi, int n_multi, const void* chunks,
                  int n_chunks, void* out, long long ldo, long long block_stride, int C, void* stream);
int dmoe_unit_recurrence(int is_f32, const DmoeUnit* d, void* stream);
// out[t, i] = act(gu[t, i]) * gu[t, I + i]; act, limit and recs as in DmoeGemm
int dmoe_gate_mul(int is_f32, int act, const void* gu, long long ld, void* out, long long ld_out, int T, int I, float limit,
                  const void* recs, void* stream);
// Y = X W^T on the CUDA cores in fp32 arithmetic: fp32 operands, or bf16 operands of any alignment.
int dmoe_simt_linear(int x_f32, int y_f32, const void* X, long long ldx, const void* W, long long ldw, void* Y, long long ldy,
                     int T, int F, int K, int act, int act_cols, void* stream);      // act 2: tanh of the output, 4: silu of its first columns
// The same over row groups: rows offs[g] .. offs[g + 1] of X with W[g] [F, K]; recs / bases (may be NULL): row t goes, scaled,
// where recs[t] says (see DmoeGemm), in X's type.
int dmoe_simt_grouped(int is_f32, int y_f32, const void* X, long long ldx, const void* W, const int* offs, int G, void* Y, long long ldy,
                      const void* recs, const void* bases, int unit_weights, int T, int F, int K, void* stream);

// ---- linear recurrences with a matrix state per head (recurrent.cu) ---------------------------------------
typedef struct DmoeRecur {
  const void* q;            // [rows, kv_heads * dim], row stride ldq; raw projections where taps > 0
  const void* k;
  const void* v;            // [rows, heads * vdim]
  const void* gate;         // [rows, heads * vdim] output gate before its activation
  const void* beta;         // delta: [rows, heads] write strength before its sigmoid
  const float* z;           // [rows, heads * dim] decay logits without their bias (kinds 0 to 2)
  const float* z_bias;      // [heads * dim]
  const float* a_log;       // [heads], decay_kind 1
  const float* conv_w;      // [2 kv_heads dim + heads vdim, taps], last column = current token
  void* ring;               // [n_slots, taps, channels]: the last inputs of the convolution, by position modulo taps
  const void* segs;         // int4 {first row, tokens, slot, first position}; NULL (decode step): segment i is row i at
  const int* positions;     // position positions[i] of the sequence in slot rows[i], skipped where kv_slots[i] < 0
  const int* rows;
  const long long* kv_slots;
  float* state;             // [n_slots, heads, dim, vdim]
  const float* norm_w;      // [vdim], or [heads, vdim] with norm_ld = vdim (0: one for all heads)
  void* out;                // [rows, heads * vdim]
  float* raw;               // read-outs before norm and gate
  long long ldq, ldk, ldv, ldg, ldb, ldz, ldo, ldraw;
  int n_segs, n_slots, heads, kv_heads, dim, vdim, taps;
  int delta;                // 0: plain write, 1: delta rule (q and k are made unit vectors)
  int decay_kind;           // 0: log a = log sigmoid(z + b) * inv_tau, 1: log a = -exp(a_log) softplus(z + b), 2: log a = -exp(z + b)
                            // 3: log a = head_decay[h]; 4: matrix memory (below)
  int gate_kind;            // 0: silu, 1: sigmoid
  int is_f32;
  int one_token;            // dmoe_recur_step: every segment has one token
  float qscale, inv_tau, eps;
  int* status;              // optional device status word: non-zero after a bounded wait gave up
  const float* bonus;       // plain write only: [heads, dim]; the read-out precedes decay and write, and the token's own write
                            // enters it weighed by the bonus of the key channel
  int norm_ld;
  const float* head_decay;  // [heads]
  // matrix memory: logs i = cap(gates[row, h] + gate_bias[h]), f = log sigmoid(cap(gates[row, heads + h] + ..)), cap(z) = gate_cap
  // tanh(z / gate_cap); running maximum m <- max(f + m, i), decay exp(f + m - m'), k scaled by exp(i - m'); read-outs are divided by
  // max(|n . q|, exp(-m)) + 1e-6, n decayed and written like a state of one value column of ones
  const float* gates;       // [rows, 2 heads], row stride ldgates
  const float* gate_bias;   // [2 heads]
  float* norm_state;        // [n_slots, heads, dim]
  float* max_state;         // [n_slots, 2, heads]: m at the parity of its position
  float* keep;              // [heads, ldsteps] log decays, factors of k and running maxima of longer segments (dmoe_memory_gates)
  float* put;
  float* run_max;
  float* scale;             // with raw: [rows, heads] factors of the read-outs (the divisions above)
  long long ldgates, ldsteps;
  float gate_cap;
} DmoeRecur;
// keep, put and run_max of the rows of a->segs; the running maxima in the slots move on.
int dmoe_memory_gates(const DmoeRecur* a, void* stream);
int dmoe_recur_value_tile(int dim, int vdim);
int dmoe_recur_step(const DmoeRecur* a, int vt, void* stream);
int dmoe_gate_norm(int is_f32, const void* table, int n, int max_tokens, const float* raw, long long ldraw, const void* gate,
                   long long ldg, const float* norm_w, int norm_ld, float eps, int gate_kind, void* out, long long ldo, int heads, int V,
                   const float* scale, void* stream);      // scale [rows, heads]: factors of the raw rows, may be NULL
// The same recurrence chunk by chunk on the tensor cores (recurrent_chunk.cu), bf16 activations, for segments of any length.
int dmoe_recur_chunk_ok(int dim, int vdim);
long long dmoe_recur_chunk_bytes(int dim, int vdim, int delta, int n_chunks);
int dmoe_recur_chunks(const DmoeRecur* a, const void* chunks, int n_chunks, void* ws, long long ws_bytes, void* stream);
int dmoe_conv_chunks(const DmoeRecur* a, const void* chunks, int n_chunks, void* out, long long ldo, void* stream);

// ---- routing (moe.cu) -------------------------------------------------------------------------------
// (RMSNorm ->) gate -> softmax -> top-k (-> renormalise); counts[e] += tokens routed to e (may be NULL).
int dmoe_route(const void* x, long long ld_x, const void* norm_w, float eps, const void* gate_w, int T, int H, int E,
               int K, int renorm, void* y, long long ld_y, int* topk_ids, float* topk_w, float* logits_out, int* counts,
               const float* logit_bias, void* stream);
int dmoe_route_ex(const void* x, long long ld_x, const void* norm_w, float eps, const void* gate_w, int T, int H, int E,
                  int K, int renorm, void* y, long long ld_y, int* topk_ids, float* topk_w, int* counts,
                  const void* add_ptrs, int n_add, long long ld_add, void* resid_out, long long ld_resid, int count_lo,
                  int count_hi, const float* logit_bias, void* stream);
// Sort-by-expert copy of the routed rows plus their 16-byte records; ws = ints [counts E | cursor E | ticket].
int dmoe_dispatch_local(const void* y, long long ld_y, const int* topk_ids, const float* topk_w, int T, int K, int H,
                        int E, int experts_per_rank, int my_rank, int* ws, int* offs, const void* x_bases,
                        long long ld_dst, const void* rec_bases, int dst_capacity, int* status, void* stream);
// The same on one device for rows of H elements of elem_bytes (2 or 4) without alignment.
int dmoe_dispatch_local_any(int elem_bytes, const void* y, long long ld_y, const int* topk_ids, const float* topk_w, int T, int K,
                            int H, int E, int* ws, int* offs, const void* x_bases, long long ld_dst, const void* rec_bases,
                            int dst_capacity, int* status, void* stream);

// ---- peer-memory dispatch (comm.cu) -----------------------------------------------------------------
// Stores every routed (token, k) row of this attention rank into its region on the expert GPU that owns the
// expert ([experts_per_rank, region_cap] rows per destination), with 16-byte records and a release flag (*epoch + 1);
// row blocks are reserved on the destinations' per-expert cursors (cnt_bases) with system-scope atomics. x_bases /
// rec_bases / cnt_bases / flag_bases are device arrays of n_dst peer pointers. ws = ints [counts E | cursor E |
// ticket, 7 pad | row_base E], counts filled by dmoe_route; cleared for the next launch.
int dmoe_dispatch_remote(const void* y, long long ld_y, const int* topk_ids, const float* topk_w, int T, int K, int H,
                         int E, int experts_per_rank, int n_dst, int my_rank, int region_cap, int* ws,
                         const void* x_bases, long long ld_dst, const void* rec_bases, const void* cnt_bases,
                         const void* flag_bases, int* epoch, int* status, int tok_lo, int tok_hi, void* stream);
// ---- fused attention-side senders (sender.cu) --------------------------------------------------------
// [wait] resid_out = resid_in + sum of n_add partial rows; y = rmsnorm(resid_out) * w is stored to row dst_row0 + t of
// EVERY buffer in dst_ptrs (device array of n_dst pointers: this GPU's and, for a tensor-parallel group, its peers'
// QKV staging buffers); then slot signal_slot of every flag array in signal_ptrs gets *signal_epoch + 1.
// The wait (flags[i] >= *wait_epoch + 1 for i < n_wait, bounded) runs inside the kernel. ticket: one zeroed int.
typedef struct DmoeNormGather {
  const void* resid_in; const void* add; const void* w; void* resid_out; const void* dst_ptrs;
  const int* wait_flags; int* wait_epoch; const void* signal_ptrs; int* signal_epoch; int* ticket; int* status;
  long long ld_in, add_row_stride, add_part_stride, ld_out, dst_row0, ld_dst;
  float eps;
  int n_add, n_dst, T, H, n_wait, n_signal, signal_slot;
} DmoeNormGather;
int dmoe_norm_gather(const DmoeNormGather* desc, void* stream);

// [wait] resid += sum of the n_add partial-row slots (add + s * add_slot_stride, row stride ld_add); y = rmsnorm(resid);
// gate -> softmax -> top-k; every (token, k) pair reserves a row in its expert's region on the owning GPU (atomic on
// cnt_bases[dst][local expert]) and stores row + record there; the last CTA sets flag_bases[d][my_rank] = *disp_epoch + 1
// for every d. gate_w == NULL: reduction and normalisation only. x_bases == NULL: route without dispatching.
typedef struct DmoeRouteDispatch {
  void* resid; const void* add; const void* norm_w; const void* gate_w; const float* logit_bias; void* y;
  int* topk_ids; float* topk_w; const void* x_bases; const void* rec_bases; const void* cnt_bases;
  const void* flag_bases; int* disp_epoch; const int* wait_flags; int* wait_epoch; int* ticket; int* status;
  long long ld_resid, add_slot_stride, ld_add, ld_y, ld_dst;
  float eps;
  int n_add, T, H, E, K, renorm, experts_per_rank, n_dst, my_rank, region_cap, n_wait;
  // rank written into the records as the owner the experts return the rows to, where that is not the sender itself
  // (pipeline-parallel attention: the stage that owns the next layer); 0 with ret_rank_set == 0 means my_rank
  int ret_rank, ret_rank_set;
} DmoeRouteDispatch;
int dmoe_route_dispatch(const DmoeRouteDispatch* desc, void* stream);
// dst_ptrs[d][dst0 + i] = src[i] (i < n) for every d < n_dst, then signal_ptrs[d][signal_slot] = *signal_epoch + 1.
int dmoe_ids_gather(const int* src, int n, const void* dst_ptrs, int n_dst, int dst0, const void* signal_ptrs,
                    int signal_slot, int* signal_epoch, void* stream);

// Waits (bounded) until flags[i] >= *epoch + 1 for i < n, then advances *epoch.
int dmoe_wait_flags(const int* flags, int n, int* epoch, int* status, void* stream);
// Cycle budget of every peer-flag wait in kernels launched from now on (<= 0: the default, about 4 s).
void dmoe_set_flag_wait_cycles(long long cycles);
int dmoe_enable_peer_access(int peer_device);
// Peer arena: a zeroed cudaMalloc block + its 64-byte CUDA IPC handle; dmoe_peer_open maps a peer's block into
// this process for kernels of the CURRENT device (peer access is enabled lazily by the driver).
int dmoe_peer_alloc(long long nbytes, void** ptr, void* handle64);
int dmoe_peer_open(const void* handle64, void** ptr);
int dmoe_peer_close(void* ptr);
int dmoe_peer_free(void* ptr);

#ifdef __cplusplus
}
#endif
