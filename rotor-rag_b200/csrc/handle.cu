// The model handle's family-independent half: position state, forwards, and the device-resident
// generation loop (the cached loop of TextGenerator, src/rotor/generation.py:179-279) with its token
// log and its captured graph.  A family (model.cu, decoder.cu) supplies the forward of a batch of token
// rows; a generation step reads the position and the input token from device memory, so one captured
// CUDA graph replays for every step.
#include "model_handle.cuh"

namespace rb {

// Cached length of every sequence: one value for all, or lens[b] when given.
__global__ void set_pos_kernel(int* pos, int n, int v, const int* lens) {
    for (int i = threadIdx.x; i < n; i += blockDim.x) pos[i] = lens ? lens[i] : v;
}

__global__ void begin_kernel(long long* cur, const long long* first, int batch, int* pos, int past, const int* lens,
                             int* step) {
    if (threadIdx.x < batch) {
        cur[threadIdx.x] = first[threadIdx.x];
        pos[threadIdx.x] = lens ? lens[threadIdx.x] : past;
    }
    if (threadIdx.x == 0) *step = 0;
}

// After a generation step: log the picked tokens and move the position on.
__global__ void advance_kernel(const long long* cur, long long* log, int batch, int max_log, int* pos, int* step) {
    const int s = *step;
    if (threadIdx.x < batch && s < max_log) log[(size_t)s * batch + threadIdx.x] = cur[threadIdx.x];
    __syncthreads();
    if (threadIdx.x < batch) pos[threadIdx.x] += 1;
    if (threadIdx.x == 0) *step = s + 1;
}

int launch_set_pos(int* pos, int n, int v, const int* lens, cudaStream_t st) {
    set_pos_kernel<<<1, 256, 0, st>>>(pos, n, v, lens);
    return launch_status();
}

int launch_advance(Model& m, const long long* picked, int batch, cudaStream_t st) {
    advance_kernel<<<1, 1024, 0, st>>>(picked, m.tok_log, batch, m.max_log, m.c.d_pos, m.d_step);
    return launch_status();
}

static int forward_family(Model& m, const long long* ids, int batch, int seq, int logits_mode, float* logits,
                          long long* next_ids, cudaStream_t st, bool advance = false) {
    return m.family->forward(m, ids, batch, seq, logits_mode, logits, next_ids, st, advance);
}

}  // namespace rb

using namespace rb;

extern "C" {

void rotor_b200_model_destroy(void* handle) {
    Model* m = (Model*)handle;
    if (!m) return;
    if (m->graph) cudaGraphExecDestroy(m->graph);
    m->family->destroy(*m);
    delete m;
}

int rotor_b200_model_forward(void* handle, const int64_t* ids, int batch, int seq, int past_len, int logits_mode,
                             float* logits, int64_t* next_ids, void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && ids && batch > 0 && seq > 0 && past_len >= 0);
    RB_REQUIRE(batch <= m->cfg.max_batch && (long)batch * seq <= m->cfg.max_rows);
    RB_REQUIRE(past_len + seq <= m->cfg.max_seq);
    RB_REQUIRE(logits_mode >= ROTOR_B200_LOGITS_NONE && logits_mode <= ROTOR_B200_LOGITS_ALL);
    RB_REQUIRE(logits_mode == ROTOR_B200_LOGITS_NONE || logits);
    cudaStream_t st = as_stream(stream);
    RB_TRY(launch_set_pos(m->c.d_pos, m->c.max_batch, past_len, nullptr, st));
    m->past = past_len;
    RB_TRY(forward_family(*m, (const long long*)ids, batch, seq, logits_mode, logits, (long long*)next_ids, st));
    m->pos = past_len + seq;
    return launch_status();
}

int rotor_b200_model_forward_rows(void* handle, const int64_t* ids, int batch, int seq, int past_len, const int32_t* rows,
                                  int nrows, float* logits, void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && ids && batch > 0 && seq > 0 && past_len >= 0 && nrows >= 0 && m->c.tp_size <= 1);
    RB_REQUIRE(batch <= m->cfg.max_batch && (long)batch * seq <= m->cfg.max_rows && past_len + seq <= m->cfg.max_seq);
    RB_REQUIRE(nrows == 0 || (rows && logits && nrows <= batch * seq));
    for (int i = 0; i < nrows; ++i) RB_REQUIRE(rows[i] >= 0 && rows[i] < batch * seq);
    cudaStream_t st = as_stream(stream);
    RB_TRY(launch_set_pos(m->c.d_pos, m->c.max_batch, past_len, nullptr, st));
    m->past = past_len;
    const int32_t none = 0;
    m->want = nrows ? rows : &none;
    m->nwant = nrows;
    const int rc = forward_family(*m, (const long long*)ids, batch, seq, nrows ? ROTOR_B200_LOGITS_ALL : ROTOR_B200_LOGITS_NONE, logits,
                              nullptr, st);
    m->want = nullptr;
    m->nwant = 0;
    if (rc) return rc;
    m->pos = past_len + seq;
    return launch_status();
}

int rotor_b200_model_decode_begin(void* handle, const int64_t* first_ids, int batch, int past_len, void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && first_ids && batch > 0 && batch <= m->cfg.max_batch && batch <= 1024);
    RB_REQUIRE(past_len >= 0 && past_len < m->cfg.max_seq);
    begin_kernel<<<1, 1024, 0, as_stream(stream)>>>(m->cur_ids, (const long long*)first_ids, batch, m->c.d_pos,
                                                    past_len, nullptr, m->d_step);
    m->pos = past_len;
    m->step = 0;
    m->batch = batch;
    return launch_status();
}

/* Prefill of a ragged batch: `ids` holds `batch` prompts right-padded to `seq` tokens (any valid
 * id as padding), lens[b] (host) the true length of prompt b, 1 <= lens[b] <= seq.  Causal
 * models only: a row then never sees the padding behind it, so every position below lens[b]
 * is what a batch-of-one forward of prompt b alone gives.  Logits / picks are taken at each
 * prompt's own last token (logits_mode NONE or LAST).  Cache positions lens[b].. hold padding
 * products; rotor_b200_model_decode_begin_ragged makes the next steps overwrite them in order. */
int rotor_b200_model_forward_ragged(void* handle, const int64_t* ids, int batch, int seq, const int32_t* lens,
                                    int logits_mode, float* logits, int64_t* next_ids, void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && ids && lens && batch > 0 && seq > 0);
    RB_REQUIRE(m->cfg.causal && m->c.tp_size <= 1);
    RB_REQUIRE(batch <= m->cfg.max_batch && (long)batch * seq <= m->cfg.max_rows && seq <= m->cfg.max_seq);
    RB_REQUIRE(logits_mode == ROTOR_B200_LOGITS_NONE || (logits_mode == ROTOR_B200_LOGITS_LAST && logits));
    for (int b = 0; b < batch; ++b) RB_REQUIRE(lens[b] >= 1 && lens[b] <= seq);
    cudaStream_t st = as_stream(stream);
    RB_TRY(launch_set_pos(m->c.d_pos, m->c.max_batch, 0, nullptr, st));
    m->past = 0;
    m->last_of = lens;
    const int rc = forward_family(*m, (const long long*)ids, batch, seq, logits_mode, logits, (long long*)next_ids, st);
    m->last_of = nullptr;
    if (rc) return rc;
    m->pos = seq;
    return launch_status();
}

/* rotor_b200_model_decode_begin for sequences of different cached lengths (host lens[b], after
 * rotor_b200_model_forward_ragged): sequence b appends at position lens[b] + step and attends
 * to its own lens[b] + step + 1 keys. */
int rotor_b200_model_decode_begin_ragged(void* handle, const int64_t* first_ids, int batch, const int32_t* lens,
                                         void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && first_ids && lens && batch > 0 && batch <= m->cfg.max_batch && batch <= 1024);
    int longest = 0;
    for (int b = 0; b < batch; ++b) {
        RB_REQUIRE(lens[b] >= 0 && lens[b] < m->cfg.max_seq);
        longest = lens[b] > longest ? lens[b] : longest;
    }
    cudaStream_t st = as_stream(stream);
    RB_CUDA(cudaMemcpyAsync(m->d_lens, lens, (size_t)batch * sizeof(int), cudaMemcpyHostToDevice, st));
    begin_kernel<<<1, 1024, 0, st>>>(m->cur_ids, (const long long*)first_ids, batch, m->c.d_pos, 0, m->d_lens,
                                     m->d_step);
    RB_CUDA(cudaStreamSynchronize(st));  // `lens` may be pageable host memory the caller reuses
    m->pos = longest;  // capacity checks follow the longest sequence
    m->step = 0;
    m->batch = batch;
    return launch_status();
}

static int one_step(Model& m, cudaStream_t st) {
    if (m.c.tp_size > 1)
        return forward_family(m, m.cur_ids, m.batch, 1, ROTOR_B200_LOGITS_NONE, nullptr, m.cur_ids, st, true);
    if (m.batch <= 4)  // pick, token log and position advance ride in the LM head's last CTA
        return forward_family(m, m.cur_ids, m.batch, 1, ROTOR_B200_LOGITS_NONE, nullptr, m.cur_ids, st, true);
    RB_TRY(forward_family(m, m.cur_ids, m.batch, 1, ROTOR_B200_LOGITS_NONE, nullptr, m.cur_ids, st));
    return launch_advance(m, m.cur_ids, m.batch, st);
}

int rotor_b200_model_decode_steps(void* handle, int nsteps, int use_graph, void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && nsteps > 0 && m->batch > 0);
    RB_REQUIRE(m->pos + nsteps <= m->cfg.max_seq && m->step + nsteps <= m->max_log);
    cudaStream_t st = as_stream(stream);
    if (!use_graph) {
        for (int i = 0; i < nsteps; ++i) RB_TRY(one_step(*m, st));
    } else {
        if (m->graph && (m->graph_batch != m->batch)) {
            cudaGraphExecDestroy(m->graph);
            m->graph = nullptr;
        }
        if (!m->graph) {
            RB_REQUIRE(st != nullptr);  // the legacy default stream cannot be captured
            cudaGraph_t g = nullptr;
            RB_CUDA(cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
            const unsigned long long before = g_launch_count;
            int rc = one_step(*m, st);
            m->graph_launches = g_launch_count - before;
            g_launch_count = before;  // captured, not run
            cudaError_t e = cudaStreamEndCapture(st, &g);
            if (rc || e != cudaSuccess) {
                if (g) cudaGraphDestroy(g);
                return rc ? rc : ROTOR_B200_ERR_CUDA;
            }
            e = cudaGraphInstantiate(&m->graph, g, 0);
            cudaGraphDestroy(g);
            if (e != cudaSuccess) return ROTOR_B200_ERR_CUDA;
            m->graph_batch = m->batch;
        }
        for (int i = 0; i < nsteps; ++i) RB_CUDA(cudaGraphLaunch(m->graph, st));
        g_launch_count += m->graph_launches * (unsigned long long)nsteps;
    }
    m->pos += nsteps;
    m->step += nsteps;
    return ROTOR_B200_OK;
}

int rotor_b200_model_read_tokens(void* handle, int first_step, int count, int64_t* tokens_host, void* stream) {
    Model* m = (Model*)handle;
    RB_REQUIRE(m && tokens_host && first_step >= 0 && count > 0 && first_step + count <= m->step);
    cudaStream_t st = as_stream(stream);
    RB_CUDA(cudaMemcpyAsync(tokens_host, m->tok_log + (size_t)first_step * m->batch,
                            (size_t)count * m->batch * sizeof(int64_t), cudaMemcpyDeviceToHost, st));
    RB_CUDA(cudaStreamSynchronize(st));
    return ROTOR_B200_OK;
}

int rotor_b200_model_position(void* handle) {
    Model* m = (Model*)handle;
    return m ? m->pos : -1;
}

}  // extern "C"
