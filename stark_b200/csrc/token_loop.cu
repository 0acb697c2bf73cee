// The token loop every model family shares: one recorded launch sequence (CUDA graph with programmatic dependent
// launch between its kernels) per token, replayed with the position and token read from device memory; prompt rows in
// batched passes; read-out, greedy chaining on the device, prefix rewind.  Mirrors the reference's decode pass
//   crates/stark-engine/src/engine/language_model/stream/stream.rs:787-1217 (one submission per token, on-device token
//   chaining) and its prefill loop (:441-686).
// What a token or a row pass launches is the family's business (ModelFamily in model.cuh).
#include <algorithm>
#include <cmath>
#include <cstring>
#include <new>
#include <vector>

#include "model.cuh"
#include "prefill.cuh"
#include "tunables.cuh"

namespace sb {

Model::~Model() {
    if (step_graph) cudaGraphExecDestroy(step_graph);
    if (ingest_graph) cudaGraphExecDestroy(ingest_graph);
    if (family && family->destroy) family->destroy(this);
    cudaFree(block_table);
    cudaFree(state);
    cudaFree(pending);
    cudaFree(generated);
    cudaFree(trace);
    cudaFree(logits);
    cudaFree(logits_f32);
    cudaFree(partial_max);
    cudaFree(partial_index);
    cudaFree(chunk_tokens);
    cudaFree(sample_scratch);
    if (host_state) cudaFreeHost(host_state);
    if (host_logits) cudaFreeHost(host_logits);
    if (stream) cudaStreamDestroy(stream);
}

// What every family's handle owns: the stream, the step state, the page table of the cache (identity, sized for the
// context in whole pages), the token lists, the logits row and its read-out buffers.
stark_b200_status model_create_session(Model *m, bool f32_logits) {
    const auto &c = m->cfg;
    stark_b200_status st;
    cudaGetDevice(&m->device);
    SB_CUDA(cudaStreamCreateWithFlags(&m->stream, cudaStreamNonBlocking));
    m->num_blocks = (c.context_tokens + kPageTokens - 1u) / kPageTokens;
    std::vector<int32_t> table(m->num_blocks);
    for (uint32_t i = 0; i < m->num_blocks; ++i) table[i] = (int32_t)i;
    if ((st = dmalloc(&m->block_table, m->num_blocks)) != STARK_B200_OK) return st;
    SB_CUDA(cudaMemcpy(m->block_table, table.data(), table.size() * 4, cudaMemcpyHostToDevice));
    if ((st = dmalloc(&m->state, 1)) != STARK_B200_OK) return st;
    if ((st = dmalloc(&m->pending, (size_t)c.context_tokens + 1u)) != STARK_B200_OK) return st;
    if ((st = dmalloc(&m->generated, (size_t)c.context_tokens + 1u)) != STARK_B200_OK) return st;
    if (f32_logits) {
        if ((st = dmalloc(&m->logits_f32, c.vocab)) != STARK_B200_OK) return st;
    } else {
        if ((st = dmalloc(&m->logits, c.vocab)) != STARK_B200_OK) return st;
    }
    if ((st = dmalloc(&m->partial_max, kLogitsPartials)) != STARK_B200_OK) return st;
    if ((st = dmalloc(&m->partial_index, kLogitsPartials)) != STARK_B200_OK) return st;
    SB_CUDA(cudaMemset(m->state, 0, sizeof(StepState)));
    if (cudaMallocHost(&m->host_state, sizeof(StepState)) != cudaSuccess ||
        cudaMallocHost(&m->host_logits, (size_t)c.vocab * (f32_logits ? 4u : 2u)) != cudaSuccess)
        return STARK_B200_OUT_OF_MEMORY;
    return STARK_B200_OK;
}

// One token on the model's stream: the recorded launch sequence, or the family's own way of running one.
static stark_b200_status launch_token(Model *m, bool full) {
    if (m->family->launch_token && m->use_mega) return m->family->launch_token(m, full);
    SB_CUDA(cudaGraphLaunch(full ? m->step_graph : m->ingest_graph, m->stream));
    return STARK_B200_OK;
}

static stark_b200_status capture(Model *m, bool full, cudaGraphExec_t *exec, uint32_t *launches) {
    SB_CUDA(cudaStreamBeginCapture(m->stream, cudaStreamCaptureModeThreadLocal));
    stark_b200_status st = m->family->issue_token(m, full, launches);
    cudaGraph_t g = nullptr;
    cudaError_t e = cudaStreamEndCapture(m->stream, &g);
    if (st != STARK_B200_OK) {
        if (g) cudaGraphDestroy(g);
        return st;
    }
    if (e != cudaSuccess) return cuda_status(e);
    e = cudaGraphInstantiate(exec, g, 0);
    cudaGraphDestroy(g);
    return cuda_status(e);
}

stark_b200_status model_finalize(Model *m) {
    if (m->finalized) return STARK_B200_INVALID_STATE;
    stark_b200_status st = m->family->ready(m);
    if (st != STARK_B200_OK) return st;
    // One eager pass first (function attributes and lazily created library state must exist before
    // a recording), on a scratch position; then record both sequences.
    if ((st = model_reset(m)) != STARK_B200_OK) return st;
    if (m->family->first_pass) {
        if ((st = m->family->first_pass(m)) != STARK_B200_OK) return st;
    } else {
        if ((st = m->family->issue_token(m, true, nullptr)) != STARK_B200_OK) return st;
        if ((st = m->family->issue_token(m, false, nullptr)) != STARK_B200_OK) return st;
    }
    SB_CUDA(cudaStreamSynchronize(m->stream));
    if ((st = capture(m, true, &m->step_graph, &m->step_launches)) != STARK_B200_OK) return st;
    if ((st = capture(m, false, &m->ingest_graph, &m->ingest_launches)) != STARK_B200_OK) return st;
    if (m->family->recorded && (st = m->family->recorded(m)) != STARK_B200_OK) return st;
    m->finalized = true;
    return model_reset(m);
}

// Records both launch sequences again with the current launch-shape settings.  Cache and position are kept.
stark_b200_status model_recapture(Model *m) {
    if (!m->finalized || m->fenced) return STARK_B200_INVALID_STATE;
    if (m->use_mega) return STARK_B200_UNSUPPORTED;
    SB_CUDA(cudaStreamSynchronize(m->stream));
    if (m->family->retune) m->family->retune(m);
    // one eager pass on a scratch copy of the step state (first use of a kernel instance sets its attributes)
    StepState saved;
    SB_CUDA(cudaMemcpy(&saved, m->state, sizeof(StepState), cudaMemcpyDeviceToHost));
    stark_b200_status st;
    if ((st = m->family->issue_token(m, true, nullptr)) != STARK_B200_OK) return st;
    if ((st = m->family->issue_token(m, false, nullptr)) != STARK_B200_OK) return st;
    SB_CUDA(cudaStreamSynchronize(m->stream));
    SB_CUDA(cudaMemcpy(m->state, &saved, sizeof(StepState), cudaMemcpyHostToDevice));
    cudaGraphExec_t step = nullptr, ingest = nullptr;
    uint32_t step_n = 0, ingest_n = 0;
    if ((st = capture(m, true, &step, &step_n)) != STARK_B200_OK) return st;
    if ((st = capture(m, false, &ingest, &ingest_n)) != STARK_B200_OK) {
        cudaGraphExecDestroy(step);
        return st;
    }
    cudaGraphExecDestroy(m->step_graph);
    cudaGraphExecDestroy(m->ingest_graph);
    m->step_graph = step;
    m->ingest_graph = ingest;
    m->step_launches = step_n;
    m->ingest_launches = ingest_n;
    m->has_logits = false;
    return STARK_B200_OK;
}

stark_b200_status model_reset(Model *m) {
    SB_CUDA(cudaMemsetAsync(m->state, 0, sizeof(StepState), m->stream));
    stark_b200_status st = m->family->reset ? m->family->reset(m) : STARK_B200_OK;
    if (st != STARK_B200_OK) return st;
    SB_CUDA(cudaStreamSynchronize(m->stream));
    m->position = 0;
    m->has_logits = false;
    return STARK_B200_OK;
}

stark_b200_status model_rewind(Model *m, uint64_t position) {
    if (position > m->position) return STARK_B200_INVALID_ARGUMENT;
    if (m->family->rewind) {
        stark_b200_status st = m->family->rewind(m, position);
        if (st != STARK_B200_OK) return st;
    }
    const uint32_t pos = (uint32_t)position;
    SB_CUDA(cudaMemcpyAsync(&m->state->position, &pos, 4, cudaMemcpyHostToDevice, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    m->position = position;
    m->has_logits = false;
    return STARK_B200_OK;
}

// Ingests `rows` prompt rows starting at position m->position (cache only: no logits).  The caller has checked
// ids and the context limit.  With a draft head loaded, every chunk also primes the head's cache with the pairs
// (next prompt token, this row's normalized hidden): dense_mtp.rs:462-584.
// `wanted` (ascending indices into ids, all < rows) are rows whose logits go to dst, [wanted_count, vocab].
static stark_b200_status prefill_batched(Model *m, const uint32_t *ids, size_t rows, size_t ids_total,
                                         const uint32_t *wanted = nullptr, size_t wanted_count = 0, float *dst = nullptr) {
    stark_b200_status st;
    size_t served = 0;
    for (size_t done = 0; done < rows; done += kPrefillBatchRows) {
        if (m->cancel_requested) return STARK_B200_CANCELLED;
        const uint32_t mrows = (uint32_t)std::min<size_t>(kPrefillBatchRows, rows - done);
        const uint32_t first_pos = (uint32_t)(m->position + done);
        // one extra id when there is one: the head's pairs need the token after each row
        const size_t upload = std::min<size_t>((size_t)mrows + 1u, ids_total - done);
        SB_CUDA(cudaMemcpyAsync(m->chunk_tokens, ids + done, upload * 4u, cudaMemcpyHostToDevice, m->stream));
        if ((st = m->family->rows_pass(m, m->chunk_tokens, mrows, first_pos)) != STARK_B200_OK) return st;
        if (m->family->rows_done && (st = m->family->rows_done(m, mrows, (uint32_t)(upload - 1u), first_pos)) != STARK_B200_OK)
            return st;
        std::vector<uint32_t> here;
        while (served + here.size() < wanted_count && wanted[served + here.size()] < done + mrows)
            here.push_back(wanted[served + here.size()] - (uint32_t)done);
        if (!here.empty()) {
            if ((st = m->family->rows_logits(m, here.data(), (uint32_t)here.size(), mrows,
                                             dst + served * m->cfg.vocab)) != STARK_B200_OK)
                return st;
            served += here.size();
        }
    }
    return STARK_B200_OK;
}

// Feeds `count` tokens; the last one runs the full sequence so that logits and the greedy token
// are available afterwards (hybrid::Model: ingest all but the last, then step the last;
// crates/stark-score/src/scoring.rs:453-489).
static stark_b200_status prefill_checked(Model *m, const uint32_t *ids, size_t count, bool batched, const uint32_t *wanted,
                                         size_t wanted_count, float *dst) {
    const ModelFamily &f = *m->family;
    if (batched) {
        // All rows but the last only fill the cache: they go through the batched path (tensor-core contraction over
        // whole chunks), after which the last row is an ordinary token at its position.
        if (f.prompt_begin) {
            stark_b200_status ps = f.prompt_begin(m, ids);
            if (ps != STARK_B200_OK) return ps;
        }
        stark_b200_status bs = prefill_batched(m, ids, count - 1, count, wanted, wanted_count, dst);
        if (bs == STARK_B200_CANCELLED) {
            m->cancel_requested = false;
            cudaStreamSynchronize(m->stream);
            model_reset(m);
            return bs;
        }
        if (bs != STARK_B200_OK) return bs;
        StepState last{};
        last.position = (uint32_t)(m->position + count - 1);
        last.token = ids[count - 1];
        SB_CUDA(cudaMemcpyAsync(m->state, &last, sizeof(last), cudaMemcpyHostToDevice, m->stream));
        stark_b200_status ls = launch_token(m, true);
        if (ls != STARK_B200_OK) return ls;
        m->position += count;
        m->has_logits = true;
        m->launches_issued += m->step_launches;
        return f.prompt_end ? f.prompt_end(m) : STARK_B200_OK;
    }
    // pending[0 .. count-2] = ids[1 ..]; the ingest-advance kernel pops one per row
    if (count > 1) SB_CUDA(cudaMemcpyAsync(m->pending, ids + 1, (count - 1) * 4, cudaMemcpyHostToDevice, m->stream));
    StepState hs{};
    hs.position = (uint32_t)m->position;
    hs.token = ids[0];
    hs.next_token = 0;
    hs.cursor = 0;
    SB_CUDA(cudaMemcpyAsync(m->state, &hs, sizeof(hs), cudaMemcpyHostToDevice, m->stream));
    for (size_t i = 0; i + 1 < count; ++i) {
        if (m->cancel_requested) {
            m->cancel_requested = false;
            cudaStreamSynchronize(m->stream);
            m->fenced = false;
            model_reset(m);
            return STARK_B200_CANCELLED;
        }
        stark_b200_status ls = launch_token(m, false);
        if (ls != STARK_B200_OK) return ls;
    }
    {
        stark_b200_status ls = launch_token(m, true);
        if (ls != STARK_B200_OK) return ls;
    }
    m->position += count;
    m->has_logits = true;
    m->launches_issued += (count - 1) * m->ingest_launches + m->step_launches;
    return STARK_B200_OK;
}

static stark_b200_status prefill_arguments(Model *m, const uint32_t *ids, size_t count) {
    if (!m->finalized || m->fenced || m->mtp.open_rows) return STARK_B200_INVALID_STATE;
    if (count == 0) return STARK_B200_INVALID_ARGUMENT;
    if (m->position + count > m->cfg.context_tokens) return STARK_B200_CONTEXT_LIMIT;
    const uint32_t vocab = m->family->input_vocab(m);
    for (size_t i = 0; i < count; ++i)
        if (ids[i] >= vocab) return STARK_B200_INVALID_ARGUMENT;
    return STARK_B200_OK;
}

static bool prefill_in_batches(Model *m, size_t count) {
    if (!tunables().prefill_batch || !m->family->rows_ready(m)) return false;
    return m->mtp.enabled || count - 1 >= std::min<size_t>(m->family->min_rows, tunables().prefill_min_rows);
}

stark_b200_status model_prefill(Model *m, const uint32_t *ids, size_t count) {
    stark_b200_status st = prefill_arguments(m, ids, count);
    if (st != STARK_B200_OK) return st;
    const bool batched = prefill_in_batches(m, count);
    if (m->mtp.enabled && (!batched || (m->position > 0 && !m->mtp.has_pending))) return STARK_B200_UNSUPPORTED;
    return prefill_checked(m, ids, count, batched, nullptr, 0, nullptr);
}

// A portion of a prompt with the logits of chosen rows.  Families that can read several rows of a pass out at once
// do; otherwise the portion is cut behind every wanted row.
stark_b200_status model_prefill_rows(Model *m, const uint32_t *ids, size_t count, const uint32_t *wanted, size_t wanted_count,
                                     float *dst) {
    stark_b200_status st = prefill_arguments(m, ids, count);
    if (st != STARK_B200_OK) return st;
    for (size_t i = 0; i < wanted_count; ++i)
        if (wanted[i] >= count || (i && wanted[i] <= wanted[i - 1])) return STARK_B200_INVALID_ARGUMENT;
    if (m->mtp.enabled) return STARK_B200_UNSUPPORTED;
    const size_t vocab = m->cfg.vocab;
    const bool last = wanted_count && wanted[wanted_count - 1] + 1u == count;
    if (prefill_in_batches(m, count) && m->family->rows_logits) {
        st = prefill_checked(m, ids, count, true, wanted, wanted_count - (last ? 1u : 0u), dst);
        if (st != STARK_B200_OK) return st;
        return last ? model_readout_f32(m, dst + (wanted_count - 1) * vocab, vocab) : STARK_B200_OK;
    }
    size_t done = 0;
    for (size_t i = 0; i <= wanted_count; ++i) {
        const size_t stop = i < wanted_count ? (size_t)wanted[i] + 1u : count;
        if (stop == done) continue;
        st = prefill_checked(m, ids + done, stop - done, prefill_in_batches(m, stop - done), nullptr, 0, nullptr);
        if (st != STARK_B200_OK) return st;
        if (i < wanted_count && (st = model_readout_f32(m, dst + i * vocab, vocab)) != STARK_B200_OK) return st;
        done = stop;
    }
    return STARK_B200_OK;
}

stark_b200_status model_step(Model *m, uint32_t token, bool chained) {
    if (!m->finalized || m->fenced || m->mtp.open_rows) return STARK_B200_INVALID_STATE;
    if (m->position + 1 > m->cfg.context_tokens) return STARK_B200_CONTEXT_LIMIT;
    if (!chained) {
        if (token >= m->family->input_vocab(m)) return STARK_B200_INVALID_ARGUMENT;
        SB_CUDA(cudaMemcpyAsync(&m->state->token, &token, 4, cudaMemcpyHostToDevice, m->stream));
    }
    {
        stark_b200_status ls = launch_token(m, true);
        if (ls != STARK_B200_OK) return ls;
    }
    m->position += 1;
    m->has_logits = true;
    m->launches_issued += m->step_launches;
    return STARK_B200_OK;
}

static stark_b200_status check_device_error(Model *m) {
    DeviceContext *ctx = device_context();
    if (!ctx) return STARK_B200_DEVICE_FAILURE;
    uint32_t word = 0;
    SB_CUDA(cudaMemcpyAsync(&word, ctx->error_word, 4, cudaMemcpyDeviceToHost, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    if (word) {
        m->fenced = true;
        return STARK_B200_DEVICE_FAILURE;
    }
    return STARK_B200_OK;
}

stark_b200_status model_drain(Model *m) {
    cudaError_t e = cudaStreamSynchronize(m->stream);
    if (e != cudaSuccess) {
        m->fenced = true;
        return cuda_status(e);
    }
    return check_device_error(m);
}

stark_b200_status model_next_token(Model *m, uint32_t *out) {
    if (!m->has_logits) return STARK_B200_INVALID_STATE;
    SB_CUDA(cudaMemcpyAsync(m->host_state, m->state, sizeof(StepState), cudaMemcpyDeviceToHost, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    *out = m->host_state->next_token;
    return STARK_B200_OK;
}

stark_b200_status model_readout_bf16(Model *m, uint16_t *dst, size_t count) {
    if (!m->has_logits) return STARK_B200_INVALID_STATE;
    if (count != m->cfg.vocab) return STARK_B200_INVALID_ARGUMENT;
    if (m->logits_f32) {
        float *host = reinterpret_cast<float *>(m->host_logits);
        SB_CUDA(cudaMemcpyAsync(host, m->logits_f32, count * 4, cudaMemcpyDeviceToHost, m->stream));
        SB_CUDA(cudaStreamSynchronize(m->stream));
        for (size_t i = 0; i < count; ++i) dst[i] = f32_to_bf16_bits(host[i]);
        return STARK_B200_OK;
    }
    SB_CUDA(cudaMemcpyAsync(m->host_logits, m->logits, count * 2, cudaMemcpyDeviceToHost, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    memcpy(dst, m->host_logits, count * 2);
    return STARK_B200_OK;
}

stark_b200_status model_readout_f32(Model *m, float *dst, size_t count) {
    if (!m->has_logits) return STARK_B200_INVALID_STATE;
    if (count != m->cfg.vocab) return STARK_B200_INVALID_ARGUMENT;
    if (m->logits_f32) {
        SB_CUDA(cudaMemcpyAsync(m->host_logits, m->logits_f32, count * 4, cudaMemcpyDeviceToHost, m->stream));
        SB_CUDA(cudaStreamSynchronize(m->stream));
        memcpy(dst, m->host_logits, count * 4);
        return STARK_B200_OK;
    }
    SB_CUDA(cudaMemcpyAsync(m->host_logits, m->logits, count * 2, cudaMemcpyDeviceToHost, m->stream));
    SB_CUDA(cudaStreamSynchronize(m->stream));
    for (size_t i = 0; i < count; ++i) dst[i] = bf16_bits_to_f32(m->host_logits[i]);
    return STARK_B200_OK;
}

// Greedy decode of `steps` tokens chained on the device: the step sequence writes its own next
// input.  Token ids come back through one small device-to-host copy per step, all asynchronous;
// the host synchronises once at the end.
stark_b200_status model_generate_greedy(Model *m, uint32_t steps, uint32_t *out_tokens) {
    if (!m->finalized || m->fenced || !m->has_logits) return STARK_B200_INVALID_STATE;
    if (m->position + steps > m->cfg.context_tokens) return STARK_B200_CONTEXT_LIMIT;
    uint32_t *pinned = nullptr;
    SB_CUDA(cudaMallocHost(&pinned, (size_t)(steps + 1u) * 4u));
    // out[0] is the token sampled from the logits already present (the prompt's last row); the
    // rest are appended to the device-side list by each step and fetched in one copy at the end.
    const uint32_t window[2] = {0u, steps};
    cudaError_t e = cudaMemcpyAsync(&pinned[0], &m->state->next_token, 4, cudaMemcpyDeviceToHost, m->stream);
    if (e == cudaSuccess) e = cudaMemcpyAsync(&m->state->gen_cursor, window, 8, cudaMemcpyHostToDevice, m->stream);
    for (uint32_t i = 0; i < steps && e == cudaSuccess; ++i) {
        if (launch_token(m, true) != STARK_B200_OK) e = last_cuda_error() != cudaSuccess ? last_cuda_error() : cudaErrorUnknown;
    }
    if (e == cudaSuccess && steps)
        e = cudaMemcpyAsync(&pinned[1], m->generated, (size_t)steps * 4u, cudaMemcpyDeviceToHost, m->stream);
    const uint32_t closed[2] = {0u, 0u};
    if (e == cudaSuccess) e = cudaMemcpyAsync(&m->state->gen_cursor, closed, 8, cudaMemcpyHostToDevice, m->stream);
    if (e == cudaSuccess) e = cudaStreamSynchronize(m->stream);
    if (e == cudaSuccess) memcpy(out_tokens, pinned, (size_t)(steps + 1u) * 4u);
    cudaFreeHost(pinned);
    if (e != cudaSuccess) {
        m->fenced = true;
        return cuda_status(e);
    }
    m->position += steps;
    m->launches_issued += (uint64_t)steps * m->step_launches;
    return check_device_error(m);
}

// Copies out the timeline slots of the launches issued since the last call and re-arms them.
stark_b200_status model_read_trace(Model *m, unsigned long long *dst, size_t count) {
    if (!m->trace) return STARK_B200_UNSUPPORTED;
    if (count != (size_t)m->trace_slots * kTraceFields) return STARK_B200_INVALID_ARGUMENT;
    SB_CUDA(cudaStreamSynchronize(m->stream));
    SB_CUDA(cudaMemcpy(dst, m->trace, count * 8u, cudaMemcpyDeviceToHost));
    std::vector<TraceSlot> init(m->trace_slots, TraceSlot{~0ull, ~0ull, 0ull, 0ull, 0ull, 0ull});
    SB_CUDA(cudaMemcpy(m->trace, init.data(), count * 8u, cudaMemcpyHostToDevice));
    return STARK_B200_OK;
}

}  // namespace sb
