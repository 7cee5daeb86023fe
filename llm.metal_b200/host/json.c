/* A small JSON reader (see json.h). */
#include "json.h"

#include <limits.h>
#include <math.h>
#include <stdlib.h>
#include <string.h>

typedef struct { const char *s; size_t n, at; } reader;

enum { MAX_DEPTH = 64 };

static void skip_space(reader *r)
{
    while (r->at < r->n && (r->s[r->at] == ' ' || r->s[r->at] == '\t' || r->s[r->at] == '\n' || r->s[r->at] == '\r')) r->at++;
}

static int take(reader *r, char c)
{
    skip_space(r);
    if (r->at < r->n && r->s[r->at] == c) { r->at++; return 1; }
    return 0;
}

static int hex4(reader *r, unsigned *out)
{
    if (r->n - r->at < 4) return -1;
    unsigned v = 0;
    for (int i = 0; i < 4; ++i) {
        const char c = r->s[r->at++];
        v = v * 16 + (c >= '0' && c <= '9' ? (unsigned)(c - '0') : c >= 'a' && c <= 'f' ? (unsigned)(c - 'a' + 10)
                      : c >= 'A' && c <= 'F' ? (unsigned)(c - 'A' + 10) : 1000000u);
        if (v >= 1000000u) return -1;
    }
    *out = v;
    return 0;
}

static size_t put_utf8(char *d, unsigned c)
{
    if (c < 0x80) { d[0] = (char)c; return 1; }
    if (c < 0x800) { d[0] = (char)(0xC0 | (c >> 6)); d[1] = (char)(0x80 | (c & 63)); return 2; }
    if (c < 0x10000) { d[0] = (char)(0xE0 | (c >> 12)); d[1] = (char)(0x80 | ((c >> 6) & 63)); d[2] = (char)(0x80 | (c & 63)); return 3; }
    d[0] = (char)(0xF0 | (c >> 18)); d[1] = (char)(0x80 | ((c >> 12) & 63)); d[2] = (char)(0x80 | ((c >> 6) & 63)); d[3] = (char)(0x80 | (c & 63));
    return 4;
}

/* A quoted string at the cursor, as a heap copy. An escape never grows: \uXXXX is six bytes, its UTF-8 at most four. */
static char *read_string(reader *r)
{
    if (!take(r, '"')) return NULL;
    size_t end = r->at;
    while (end < r->n && r->s[end] != '"') end += r->s[end] == '\\' ? 2 : 1;
    if (end >= r->n) return NULL;
    char *out = malloc(end - r->at + 1), *d = out;
    if (!out) return NULL;
    while (r->at < end) {
        char c = r->s[r->at++];
        if ((unsigned char)c < 0x20) { free(out); return NULL; }
        if (c != '\\') { *d++ = c; continue; }
        c = r->s[r->at++];
        unsigned u, lo;
        switch (c) {
        case '"': case '\\': case '/': *d++ = c; break;
        case 'b': *d++ = '\b'; break;
        case 'f': *d++ = '\f'; break;
        case 'n': *d++ = '\n'; break;
        case 'r': *d++ = '\r'; break;
        case 't': *d++ = '\t'; break;
        case 'u':
            if (hex4(r, &u)) { free(out); return NULL; }
            if (u >= 0xD800 && u < 0xDC00 && r->n - r->at >= 6 && r->s[r->at] == '\\' && r->s[r->at + 1] == 'u') {
                r->at += 2;
                if (hex4(r, &lo) || lo < 0xDC00 || lo > 0xDFFF) { free(out); return NULL; }
                u = 0x10000 + ((u - 0xD800) << 10) + (lo - 0xDC00);
            }
            d += put_utf8(d, u);
            break;
        default: free(out); return NULL;
        }
    }
    *d = 0;
    r->at = end + 1;
    return out;
}

static json *read_value(reader *r, int depth);

static int read_members(reader *r, json *v, int object, int depth)
{
    const char close = object ? '}' : ']';
    json **tail = &v->child;
    if (take(r, close)) return 0;
    do {
        char *key = NULL;
        if (object && (!(key = read_string(r)) || !take(r, ':'))) { free(key); return -1; }
        json *m = read_value(r, depth + 1);
        if (!m) { free(key); return -1; }
        m->key = key;
        *tail = m;
        tail = &m->next;
        v->n++;
    } while (take(r, ','));
    return take(r, close) ? 0 : -1;
}

static json *read_value(reader *r, int depth)
{
    skip_space(r);
    if (depth > MAX_DEPTH || r->at >= r->n) return NULL;
    json *v = calloc(1, sizeof(*v));
    if (!v) return NULL;
    const char c = r->s[r->at];
    const size_t left = r->n - r->at;
    int bad = 0;
    if (c == '{' || c == '[') {
        r->at++;
        v->type = c == '{' ? JSON_OBJECT : JSON_ARRAY;
        bad = read_members(r, v, c == '{', depth);
    } else if (c == '"') {
        v->type = JSON_STRING;
        bad = (v->string = read_string(r)) == NULL;
    } else if (left >= 4 && !memcmp(r->s + r->at, "true", 4)) {
        v->type = JSON_BOOL; v->number = 1; r->at += 4;
    } else if (left >= 5 && !memcmp(r->s + r->at, "false", 5)) {
        v->type = JSON_BOOL; r->at += 5;
    } else if (left >= 4 && !memcmp(r->s + r->at, "null", 4)) {
        r->at += 4;
    } else {
        char buf[64];
        size_t k = 0;
        while (k < left && k < sizeof(buf) - 1 && r->s[r->at + k] && strchr("+-0123456789.eE", r->s[r->at + k])) { buf[k] = r->s[r->at + k]; ++k; }
        buf[k] = 0;
        char *end = buf;
        v->type = JSON_NUMBER;
        v->number = strtod(buf, &end);
        bad = k == 0 || *end != 0;
        r->at += k;
    }
    if (bad) { json_free(v); return NULL; }
    return v;
}

json *json_parse(const char *text, size_t len, size_t *error_at)
{
    reader r = {text, len, 0};
    json *v = read_value(&r, 0);
    skip_space(&r);
    if (v && r.at != len) { json_free(v); v = NULL; }
    if (error_at) *error_at = r.at;
    return v;
}

void json_free(json *v)
{
    while (v) {
        json *next = v->next;
        json_free(v->child);
        free(v->string);
        free(v->key);
        free(v);
        v = next;
    }
}

const json *json_get(const json *object, const char *key)
{
    if (!object || object->type != JSON_OBJECT) return NULL;
    for (const json *m = object->child; m; m = m->next)
        if (!strcmp(m->key, key)) return m;
    return NULL;
}

int json_number(const json *object, const char *key, double *out)
{
    const json *m = json_get(object, key);
    if (!m || m->type != JSON_NUMBER) return -1;
    *out = m->number;
    return 0;
}

int json_int(const json *object, const char *key, int *out)
{
    double d;
    if (json_number(object, key, &d) || d != floor(d) || d < INT_MIN || d > INT_MAX) return -1;
    *out = (int)d;
    return 0;
}

const char *json_string(const json *object, const char *key)
{
    const json *m = json_get(object, key);
    return m && m->type == JSON_STRING ? m->string : NULL;
}
